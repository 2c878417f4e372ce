// The seam between two layers of a decoder with an fp32 residual stream: one kernel adds what the last layer's
// branches produced and writes the normalised input of every branch of the next layer.
//
//   x      = table[ids[t]] * scale                      (first layer: the embedding), or
//   x[t]  += a[t] + (b[t] or sum_k pair_w * e[inverse[t, k]])     (mixer branch, feed-forward branch)
//   n1[t]  = x[t] / rms(x[t]) * w1                      (input of one branch)
//   n2     = x[t] / rms(x[t]) * w2                      (input of a parallel branch with its own norm weight)
//
// `e` holds expert outputs in expert order, so a mixture-of-experts feed-forward needs no combine kernel; n2 can be
// written straight into expert order (`scatter` [T, k2]: the rows token t occupies), so it needs no permute kernel
// either. `rows` restricts the kernel to some rows of x (the ones whose logits are wanted).
//
// A second kernel serves layers whose two mixer branches have output norms of their own and whose update is scaled:
//
//   x[t]  += mult * (ab_scale * (a / rms(a) * norm_a + b / rms(b) * norm_b) + c)
//            [+ inject_scale * inject[ids[t]]] [+ step]       (what a looped pass adds before its first layer)
//
// A third one serves layers that norm a branch before and after it (sandwich norms), with layer norms or RMS norms:
//
//   x[t]  += mult * norm(u[t]; w_u, b_u),   n1[t] = norm(x[t]; w1, b1),   u = a[t] or sum_k pair_w[t, k] e[inverse[t, k]]
//
// with the embedding (and rows of a second table, chosen by ids of their own) ahead of the first layer. A row lives in
// registers from its first read to its last write. Every warp takes the mean and the squared deviations of its own values, and
// the parts of the warps are put together (counts, means, deviations), so a norm costs one barrier.
//
// Also here: tanh-GELU in place, the sigmoid output gate of an attention layer and the soft cap of logits.
#include <cuda_runtime.h>

#include "../common/api.h"
#include "../common/launch.h"
#include "../common/scalar.cuh"

namespace mb {
namespace resnorm {

template <typename T>
struct Params {
  float* x;
  int ldx;
  const int64_t* ids;
  const T* table;
  float scale;
  int vocab, ld_table;
  const T* a;
  int lda;
  const T* b;
  int ldb;
  const T* e;
  int lde;
  const int32_t* inverse;
  int top_k;
  float pair_w;
  const int32_t* rows;
  const T* w1;
  T* n1;
  int ld1;
  const T* w2;
  T* n2;
  int ld2;
  const int32_t* scatter;
  int k2;
  int cols, cols_pad, store_x;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(1024) residual_norm_kernel(const Params<T> p) {
  extern __shared__ float4 row_cache[];   // the updated row
  __shared__ float part[32];
  __shared__ int32_t pos_in[32], pos_out[32];
  const int out_row = blockIdx.x;
  const int row = p.rows ? p.rows[out_row] : out_row;
  float* xr = p.x + static_cast<size_t>(row) * p.ldx;
  const T* er = nullptr;
  bool have_id = true;
  if (p.table) {
    const int64_t id = p.ids[row];
    have_id = id >= 0 && id < p.vocab;
    er = p.table + static_cast<size_t>(have_id ? id : 0) * p.ld_table;
  }
  const int nvec = p.cols_pad >> 2;
  float ss = 0.f;
  // the expert rows of this token, read once
  const bool cached_in = p.e && p.top_k <= 32, cached_out = p.scatter && p.k2 <= 32;
  if (cached_in && threadIdx.x < p.top_k) pos_in[threadIdx.x] = p.inverse[static_cast<size_t>(row) * p.top_k + threadIdx.x];
  if (cached_out && threadIdx.x < p.k2) pos_out[threadIdx.x] = p.scatter[static_cast<size_t>(row) * p.k2 + threadIdx.x];
  if (cached_in || cached_out) __syncthreads();
  for (int v = threadIdx.x; v < nvec; v += blockDim.x) {
    const int c = v * 4;
    float4 x;
    if (p.table) {
      x = have_id ? ld4(er + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      x.x *= p.scale; x.y *= p.scale; x.z *= p.scale; x.w *= p.scale;
    } else {
      x = *reinterpret_cast<const float4*>(xr + c);
    }
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    if (p.e) {
#pragma unroll 4
      for (int k = 0; k < p.top_k; ++k) {
        const int pos = cached_in ? pos_in[k] : p.inverse[static_cast<size_t>(row) * p.top_k + k];
        if (pos < 0) continue;
        const float4 y = ld4(p.e + static_cast<size_t>(pos) * p.lde + c);
        s.x = fmaf(p.pair_w, y.x, s.x); s.y = fmaf(p.pair_w, y.y, s.y);
        s.z = fmaf(p.pair_w, y.z, s.z); s.w = fmaf(p.pair_w, y.w, s.w);
      }
    } else if (p.b) {
      s = ld4(p.b + static_cast<size_t>(row) * p.ldb + c);
    }
    if (p.a) {
      const float4 y = ld4(p.a + static_cast<size_t>(row) * p.lda + c);
      s.x += y.x; s.y += y.y; s.z += y.z; s.w += y.w;
    }
    x.x += s.x; x.y += s.y; x.z += s.z; x.w += s.w;
    if (p.store_x) *reinterpret_cast<float4*>(xr + c) = x;
    ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
    row_cache[v] = x;
  }
  if (p.w1 == nullptr) return;
  ss = warp_allsum(ss);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < static_cast<int>(blockDim.x >> 5); ++i) tot += part[i];
  const float inv = 1.f / sqrtf(tot / static_cast<float>(p.cols) + p.eps);
  T* o1 = p.n1 + static_cast<size_t>(out_row) * p.ld1;
  for (int v = threadIdx.x; v < nvec; v += blockDim.x) {
    const int c = v * 4;
    float4 x = row_cache[v];
    x.x *= inv; x.y *= inv; x.z *= inv; x.w *= inv;
    const float4 w = ld4(p.w1 + c);
    st4(o1 + c, make_float4(x.x * w.x, x.y * w.y, x.z * w.z, x.w * w.w));
    if (p.w2) {
      const float4 u = ld4(p.w2 + c);
      const float4 y = make_float4(x.x * u.x, x.y * u.y, x.z * u.z, x.w * u.w);
      if (p.scatter) {
        for (int k = 0; k < p.k2; ++k) {
          const int pos = cached_out ? pos_out[k] : p.scatter[static_cast<size_t>(row) * p.k2 + k];
          if (pos >= 0) st4(p.n2 + static_cast<size_t>(pos) * p.ld2 + c, y);
        }
      } else {
        st4(p.n2 + static_cast<size_t>(out_row) * p.ld2 + c, y);
      }
    }
  }
}

template <typename T>
struct MixParams {
  const T *norm_a, *norm_b, *c, *inject, *step;
  int ldc, ld_inject;
  float ab_scale, mult, inject_scale;
};

__device__ __forceinline__ float sq4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// sums of `N` values per thread over the CTA
template <int N>
__device__ __forceinline__ void block_sums(float (&v)[N], float (*part)[32]) {
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = warp_allsum(v[i]);
  if ((threadIdx.x & 31) == 0)
#pragma unroll
    for (int i = 0; i < N; ++i) part[i][threadIdx.x >> 5] = v[i];
  __syncthreads();
#pragma unroll
  for (int i = 0; i < N; ++i) {
    v[i] = 0.f;
    for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) v[i] += part[i][w];
  }
}

template <typename T>
__global__ void __launch_bounds__(1024) branch_norm_kernel(const Params<T> p, const MixParams<T> m) {
  extern __shared__ float4 row_cache[];   // the updated row
  __shared__ float part[2][32], part2[1][32];
  const int out_row = blockIdx.x;
  const int row = p.rows ? p.rows[out_row] : out_row;
  float* xr = p.x + static_cast<size_t>(row) * p.ldx;
  const T *ar = p.a ? p.a + static_cast<size_t>(row) * p.lda : nullptr, *br = p.b ? p.b + static_cast<size_t>(row) * p.ldb : nullptr;
  const T* cr = m.c ? m.c + static_cast<size_t>(row) * m.ldc : nullptr;
  const T *er = nullptr, *ir = nullptr;
  if (p.table || m.inject) {
    const int64_t id = p.ids[row];
    if (id >= 0 && id < p.vocab) {
      if (p.table) er = p.table + static_cast<size_t>(id) * p.ld_table;
      if (m.inject) ir = m.inject + static_cast<size_t>(id) * m.ld_inject;
    }
  }
  const int nvec = p.cols_pad >> 2;
  float inv_a = 1.f, inv_b = 1.f;
  if (m.norm_a || m.norm_b) {
    float s[2] = {0.f, 0.f};
    for (int v = threadIdx.x; v < nvec; v += blockDim.x) {
      if (m.norm_a) s[0] += sq4(ld4(ar + v * 4));
      if (m.norm_b) s[1] += sq4(ld4(br + v * 4));
    }
    block_sums(s, part);
    inv_a = 1.f / sqrtf(s[0] / static_cast<float>(p.cols) + p.eps);
    inv_b = 1.f / sqrtf(s[1] / static_cast<float>(p.cols) + p.eps);
  }
  float ss[1] = {0.f};
  for (int v = threadIdx.x; v < nvec; v += blockDim.x) {
    const int c = v * 4;
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f), u = x;
    if (p.table) {
      if (er) { x = ld4(er + c); x.x *= p.scale; x.y *= p.scale; x.z *= p.scale; x.w *= p.scale; }
    } else {
      x = *reinterpret_cast<const float4*>(xr + c);
    }
    auto branch = [&](const T* src, const T* w, float inv) {
      float4 y = ld4(src + c);
      if (w) {
        const float4 g = ld4(w + c);
        y.x *= inv * g.x; y.y *= inv * g.y; y.z *= inv * g.z; y.w *= inv * g.w;
      }
      u.x = fmaf(m.ab_scale, y.x, u.x); u.y = fmaf(m.ab_scale, y.y, u.y);
      u.z = fmaf(m.ab_scale, y.z, u.z); u.w = fmaf(m.ab_scale, y.w, u.w);
    };
    if (ar) branch(ar, m.norm_a, inv_a);
    if (br) branch(br, m.norm_b, inv_b);
    if (cr) { const float4 y = ld4(cr + c); u.x += y.x; u.y += y.y; u.z += y.z; u.w += y.w; }
    x.x = fmaf(m.mult, u.x, x.x); x.y = fmaf(m.mult, u.y, x.y); x.z = fmaf(m.mult, u.z, x.z); x.w = fmaf(m.mult, u.w, x.w);
    if (ir) {
      const float4 y = ld4(ir + c);
      x.x = fmaf(m.inject_scale, y.x, x.x); x.y = fmaf(m.inject_scale, y.y, x.y);
      x.z = fmaf(m.inject_scale, y.z, x.z); x.w = fmaf(m.inject_scale, y.w, x.w);
    }
    if (m.step) { const float4 y = ld4(m.step + c); x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w; }
    if (p.store_x) *reinterpret_cast<float4*>(xr + c) = x;
    ss[0] += sq4(x);
    row_cache[v] = x;
  }
  if (p.w1 == nullptr) return;
  block_sums(ss, part2);
  const float inv = 1.f / sqrtf(ss[0] / static_cast<float>(p.cols) + p.eps);
  T *o1 = p.n1 + static_cast<size_t>(out_row) * p.ld1, *o2 = p.w2 ? p.n2 + static_cast<size_t>(out_row) * p.ld2 : nullptr;
  for (int v = threadIdx.x; v < nvec; v += blockDim.x) {
    const int c = v * 4;
    float4 x = row_cache[v];
    x.x *= inv; x.y *= inv; x.z *= inv; x.w *= inv;
    const float4 w = ld4(p.w1 + c);
    st4(o1 + c, make_float4(x.x * w.x, x.y * w.y, x.z * w.z, x.w * w.w));
    if (o2) {
      const float4 g = ld4(p.w2 + c);
      st4(o2 + c, make_float4(x.x * g.x, x.y * g.y, x.z * g.z, x.w * g.w));
    }
  }
}

template <typename T>
static int run(const MbResidualNorm& q, cudaStream_t stream) {
  Params<T> p;
  p.x = q.x; p.ldx = q.ldx;
  p.ids = q.ids; p.table = static_cast<const T*>(q.table); p.scale = q.scale; p.vocab = q.vocab; p.ld_table = q.ld_table;
  p.a = static_cast<const T*>(q.a); p.lda = q.lda;
  p.b = static_cast<const T*>(q.b); p.ldb = q.ldb;
  p.e = static_cast<const T*>(q.e); p.lde = q.lde; p.inverse = q.inverse; p.top_k = q.top_k; p.pair_w = q.pair_w;
  p.rows = q.rows;
  p.w1 = static_cast<const T*>(q.w1); p.n1 = static_cast<T*>(q.n1); p.ld1 = q.ld1;
  p.w2 = static_cast<const T*>(q.w2); p.n2 = static_cast<T*>(q.n2); p.ld2 = q.ld2;
  p.scatter = q.scatter; p.k2 = q.k2;
  p.cols = q.cols; p.cols_pad = q.cols_pad; p.store_x = q.store_x; p.eps = q.eps;
  const int nvec = p.cols_pad / 4;
  // few rows: one pass per row with as many threads as it has vectors; many rows: small CTAs, several per SM
  const int most = q.n_rows <= 296 ? 1024 : 256;
  const int threads = nvec >= most ? most : (nvec + 31) / 32 * 32;
  if (q.norm_a || q.norm_b || q.c || q.inject || q.step || q.mult != 1.f || q.ab_scale != 1.f) {
    if (q.e || q.scatter || (q.norm_a && !q.a) || (q.norm_b && !q.b)) return MB_ERR_SHAPE;
    MixParams<T> m = {static_cast<const T*>(q.norm_a), static_cast<const T*>(q.norm_b), static_cast<const T*>(q.c),
                      static_cast<const T*>(q.inject), static_cast<const T*>(q.step), q.ldc, q.ld_inject, q.ab_scale, q.mult,
                      q.inject_scale};
    return launch_plain(branch_norm_kernel<T>, dim3(q.n_rows), dim3(threads), static_cast<size_t>(p.cols_pad) * 4, stream, p, m) ==
                   cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
  }
  return launch_plain(residual_norm_kernel<T>, dim3(q.n_rows), dim3(threads), static_cast<size_t>(p.cols_pad) * 4, stream, p) ==
                 cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

// ---- sandwich norms
// count, mean and sum of squared deviations of some values
struct Part {
  float n, mean, m2;
};

template <typename T, int NV, bool CENTER>
__global__ void __launch_bounds__(1024) sandwich_norm_kernel(const MbSandwichNorm p) {
  __shared__ float sums[2][32];
  __shared__ Part parts[2][32];
  __shared__ int32_t pos[32];
  __shared__ float pw[32];
  const int out_row = blockIdx.x, nvec = p.cols_pad >> 2;
  const int row = p.rows ? p.rows[out_row] : out_row;
  float* xr = p.x + static_cast<size_t>(row) * p.ldx;
  const T *ar = p.a ? static_cast<const T*>(p.a) + static_cast<size_t>(row) * p.lda : nullptr, *er = nullptr, *ir = nullptr;
  const T* ee = static_cast<const T*>(p.e);
  if (p.table) {
    const int64_t id = p.ids[row];
    if (id >= 0 && id < p.vocab) er = static_cast<const T*>(p.table) + static_cast<size_t>(id) * p.ld_table;
  }
  if (p.inject) {
    const int64_t id = p.inject_ids[row];
    if (id >= 0 && id < p.inject_rows) ir = static_cast<const T*>(p.inject) + static_cast<size_t>(id) * p.ld_inject;
  }
  if (ee && threadIdx.x < p.top_k) {
    pos[threadIdx.x] = p.inverse[static_cast<size_t>(row) * p.top_k + threadIdx.x];
    pw[threadIdx.x] = p.pair_w[static_cast<size_t>(row) * p.top_k + threadIdx.x];
  }
  float4 x[NV], u[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * blockDim.x, c = v * 4;
    x[i] = u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (v >= nvec) continue;
    if (!p.table) x[i] = *reinterpret_cast<const float4*>(xr + c);
    else if (er) { const float4 y = ld4(er + c); x[i] = make_float4(y.x * p.scale, y.y * p.scale, y.z * p.scale, y.w * p.scale); }
    if (ir) { const float4 y = ld4(ir + c); x[i].x += y.x; x[i].y += y.y; x[i].z += y.z; x[i].w += y.w; }
    if (ar) u[i] = ld4(ar + c);
  }
  if (ee) {
    __syncthreads();
#pragma unroll 4
    for (int k = 0; k < p.top_k; ++k) {
      const int at = pos[k];
      if (at < 0) continue;
      const float w = pw[k];
      const T* src = ee + static_cast<size_t>(at) * p.lde;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v >= nvec) continue;
        const float4 y = ld4(src + v * 4);
        u[i].x = fmaf(w, y.x, u[i].x); u[i].y = fmaf(w, y.y, u[i].y);
        u[i].z = fmaf(w, y.z, u[i].z); u[i].w = fmaf(w, y.w, u[i].w);
      }
    }
  }
  // r becomes the deviations from its mean (CENTER; zero beyond the true width); the result is 1 / sqrt(mean of squares + eps)
  auto scale_of = [&](float4 (&r)[NV], int stage) {
    const float n = static_cast<float>(p.cols);
    if (!CENTER) {
      float q[1] = {0.f};
#pragma unroll
      for (int i = 0; i < NV; ++i) q[0] += sq4(r[i]);
      block_sums(q, &sums[stage]);
      return 1.f / sqrtf(q[0] / n + p.eps);
    }
    // deviations from the mean of this warp's values first
    float sum = 0.f, count = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      sum += (r[i].x + r[i].y) + (r[i].z + r[i].w);                          // padding holds zeros
      const int c = ((threadIdx.x & ~31) + i * blockDim.x) * 4;              // the warp's 128 columns
      count += static_cast<float>(min(max(p.cols - c, 0), 128));
    }
    sum = warp_allsum(sum);
    float mean = count > 0.f ? sum / count : 0.f, m2 = 0.f;
    auto shift = [&](float by) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (threadIdx.x + i * blockDim.x) * 4;
        if (c + 3 < p.cols) {
          r[i].x -= by; r[i].y -= by; r[i].z -= by; r[i].w -= by;
        } else if (c < p.cols) {
          r[i].x -= by;
          if (c + 1 < p.cols) r[i].y -= by;
          if (c + 2 < p.cols) r[i].z -= by;
        }
      }
    };
    shift(mean);
#pragma unroll
    for (int i = 0; i < NV; ++i) m2 += sq4(r[i]);
    m2 = warp_allsum(m2);
    const int warps = blockDim.x >> 5;
    if (warps > 1) {                                                         // then the warps' parts together
      if ((threadIdx.x & 31) == 0) parts[stage][threadIdx.x >> 5] = Part{count, mean, m2};
      __syncthreads();
      const int lane = threadIdx.x & 31;
      Part a = {0.f, 0.f, 0.f};
      if (lane < warps) a = parts[stage][lane];
      const float all = warp_allsum(a.n * a.mean) / n;
      m2 = warp_allsum(fmaf(a.n * (a.mean - all), a.mean - all, a.m2));
      shift(all - mean);
    }
    return 1.f / sqrtf(m2 / n + p.eps);
  };
  auto affine = [&](float4 r, float inv, const void* w, const void* b, int c) {
    const float4 g = ld4(static_cast<const T*>(w) + c);
    float4 y = make_float4(r.x * inv * g.x, r.y * inv * g.y, r.z * inv * g.z, r.w * inv * g.w);
    if (CENTER) { const float4 o = ld4(static_cast<const T*>(b) + c); y.x += o.x; y.y += o.y; y.z += o.z; y.w += o.w; }
    return y;
  };
  if (ar || ee) {
    const float inv = p.w_u ? scale_of(u, 0) : 1.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v >= nvec) continue;
      const float4 y = p.w_u ? affine(u[i], inv, p.w_u, p.b_u, v * 4) : u[i];
      x[i].x = fmaf(p.mult, y.x, x[i].x); x[i].y = fmaf(p.mult, y.y, x[i].y);
      x[i].z = fmaf(p.mult, y.z, x[i].z); x[i].w = fmaf(p.mult, y.w, x[i].w);
    }
  }
  if (p.store_x) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v < nvec) *reinterpret_cast<float4*>(xr + v * 4) = x[i];
    }
  }
  if (!p.w1) return;
  const float inv = scale_of(x, 1);
  T* o1 = static_cast<T*>(p.n1) + static_cast<size_t>(out_row) * p.ld1;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v < nvec) st4(o1 + v * 4, affine(x[i], inv, p.w1, p.b1, v * 4));
  }
}

template <typename T, bool CENTER>
static int run_sandwich(const MbSandwichNorm& p, cudaStream_t stream) {
  const int nvec = p.cols_pad / 4;
  // few rows: as many threads as a row has vectors; many rows: small CTAs, several per SM
  const int most = p.n_rows <= 296 ? 1024 : 256, warps = (nvec + 31) / 32;
  int nv = (nvec + most - 1) / most;
  nv = nv <= 1 ? 1 : nv <= 2 ? 2 : 4;
  const int threads = (warps + nv - 1) / nv * 32;
  if (threads > 1024) return MB_ERR_TOO_LARGE;
  cudaError_t e;
  if (nv == 1) e = launch_plain(sandwich_norm_kernel<T, 1, CENTER>, dim3(p.n_rows), dim3(threads), 0, stream, p);
  else if (nv == 2) e = launch_plain(sandwich_norm_kernel<T, 2, CENTER>, dim3(p.n_rows), dim3(threads), 0, stream, p);
  else e = launch_plain(sandwich_norm_kernel<T, 4, CENTER>, dim3(p.n_rows), dim3(threads), 0, stream, p);
  return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

__global__ void bigram_rows_kernel(const int64_t* __restrict__ tokens, const int32_t* __restrict__ q_start,
                                   const int32_t* __restrict__ q_len, const int32_t* __restrict__ kv_len,
                                   const int32_t* __restrict__ state_idx, int64_t* __restrict__ last, int64_t* __restrict__ out, int T,
                                   int B, long long mul_prev, long long mul_cur, long long buckets) {
  const int t = blockIdx.x * blockDim.x + threadIdx.x;
  if (t >= T) return;
  int lo = 0, hi = B - 1;                       // the last sequence that starts at or before t
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (q_start[mid] <= t) lo = mid; else hi = mid - 1;
  }
  const int off = t - q_start[lo], n = q_len[lo];
  if (off < 0 || off >= n) { out[t] = buckets; return; }   // a row of no sequence
  const long long cur = tokens[t];
  long long prev = -1;
  if (off > 0) {
    prev = tokens[t - 1];
  } else {                                      // one thread per sequence reads its slot and then advances it
    const int slot = state_idx[lo];
    if (slot >= 0) {
      if (kv_len[lo] > n) prev = last[slot];
      last[slot] = tokens[t + n - 1];
    }
  }
  long long r = prev < 0 ? buckets : (prev * mul_prev + cur * mul_cur) % buckets;
  out[t] = r < 0 ? r + buckets : r;
}

template <typename T>
__global__ void gelu_tanh_kernel(T* __restrict__ x, size_t n4) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n4) return;
  const float4 v = ld4(x + i * 4);
  auto f = [](float z) { return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); };
  st4(x + i * 4, make_float4(f(v.x), f(v.y), f(v.z), f(v.w)));
}

__global__ void softcap_kernel(float* __restrict__ x, size_t n, float cap) {
  const size_t i = (static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x) * 4;
  if (i + 4 <= n) {
    float4 v = *reinterpret_cast<const float4*>(x + i);
    v.x = cap * tanhf(v.x / cap); v.y = cap * tanhf(v.y / cap); v.z = cap * tanhf(v.z / cap); v.w = cap * tanhf(v.w / cap);
    *reinterpret_cast<float4*>(x + i) = v;
  } else {
    for (size_t j = i; j < n; ++j) x[j] = cap * tanhf(x[j] / cap);
  }
}

// o[r, c] *= sigmoid(g[r, c])
template <typename T>
__global__ void sigmoid_gate_kernel(T* __restrict__ o, int ldo, const T* __restrict__ g, int ldg, int rows, int cols4) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= static_cast<size_t>(rows) * cols4) return;
  const int r = static_cast<int>(i / cols4), c = static_cast<int>(i % cols4) * 4;
  T* po = o + static_cast<size_t>(r) * ldo + c;
  const float4 a = ld4(po), b = ld4(g + static_cast<size_t>(r) * ldg + c);
  st4(po, make_float4(a.x * sigmoidf(b.x), a.y * sigmoidf(b.y), a.z * sigmoidf(b.z), a.w * sigmoidf(b.w)));
}

}  // namespace resnorm
}  // namespace mb

using namespace mb;
using namespace mb::resnorm;

extern "C" int mb_residual_norm(const MbResidualNorm* q, int dtype, cudaStream_t stream) {
  if (q->n_rows <= 0) return MB_OK;
  if (q->cols <= 0 || q->cols > q->cols_pad || q->cols_pad % 4 || q->ldx % 4 || q->lda % 4 || q->ldb % 4 || q->lde % 4 ||
      q->ld1 % 4 || q->ld2 % 4 || q->ld_table % 4 || q->ldc % 4 || q->ld_inject % 4)
    return MB_ERR_SHAPE;
  if (q->cols_pad > 12288) return MB_ERR_TOO_LARGE;
  return dtype == kF32 ? run<float>(*q, stream) : run<__nv_bfloat16>(*q, stream);
}

extern "C" int mb_sandwich_norm(const MbSandwichNorm* q, int dtype, cudaStream_t stream) {
  if (q->n_rows <= 0) return MB_OK;
  if (q->cols <= 0 || q->cols > q->cols_pad || q->cols_pad % 4 || q->ldx % 4 || q->lda % 4 || q->lde % 4 || q->ld1 % 4 ||
      q->ld_table % 4 || q->ld_inject % 4 || (q->a && q->e) || (q->e && (q->top_k <= 0 || q->top_k > 32)) ||
      (q->w_u && q->w1 && (q->b_u == nullptr) != (q->b1 == nullptr)))
    return MB_ERR_SHAPE;
  const bool center = q->b_u != nullptr || q->b1 != nullptr;
  if (dtype == kF32) return center ? run_sandwich<float, true>(*q, stream) : run_sandwich<float, false>(*q, stream);
  return center ? run_sandwich<__nv_bfloat16, true>(*q, stream) : run_sandwich<__nv_bfloat16, false>(*q, stream);
}

extern "C" int mb_bigram_rows(const int64_t* tokens, const int32_t* q_start, const int32_t* q_len, const int32_t* kv_len,
                              const int32_t* state_idx, int64_t* last, int64_t* out, int T, int B, long long mul_prev,
                              long long mul_cur, long long buckets, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return MB_OK;
  if (buckets <= 0) return MB_ERR_SHAPE;
  return launch_plain(bigram_rows_kernel, dim3((T + 255) / 256), dim3(256), 0, stream, tokens, q_start, q_len, kv_len, state_idx, last,
                      out, T, B, mul_prev, mul_cur, buckets) == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

extern "C" int mb_gelu_tanh(void* x, long long n, int dtype, cudaStream_t stream) {
  if (n <= 0) return MB_OK;
  if (n % 4) return MB_ERR_SHAPE;
  const size_t n4 = static_cast<size_t>(n) / 4;
  const dim3 grid(static_cast<unsigned>((n4 + 255) / 256));
  cudaError_t e = dtype == kF32 ? launch_plain(gelu_tanh_kernel<float>, grid, dim3(256), 0, stream, static_cast<float*>(x), n4)
                                : launch_plain(gelu_tanh_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream,
                                           static_cast<__nv_bfloat16*>(x), n4);
  return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

extern "C" int mb_softcap(float* x, long long n, float cap, cudaStream_t stream) {
  if (n <= 0) return MB_OK;
  if (!(cap > 0.f)) return MB_ERR_SHAPE;
  if (reinterpret_cast<uintptr_t>(x) & 15) return MB_ERR_ALIGN;
  const dim3 grid(static_cast<unsigned>((n + 1023) / 1024));
  return launch_plain(softcap_kernel, grid, dim3(256), 0, stream, x, static_cast<size_t>(n), cap) == cudaSuccess ? MB_OK
                                                                                                                 : MB_ERR_LAUNCH;
}

extern "C" int mb_sigmoid_gate(void* o, int ldo, const void* g, int ldg, int rows, int cols, int dtype,
                               cudaStream_t stream) {
  if (rows <= 0) return MB_OK;
  if (cols % 4 || ldo % 4 || ldg % 4) return MB_ERR_SHAPE;
  const int c4 = cols / 4;
  const dim3 grid(static_cast<unsigned>((static_cast<size_t>(rows) * c4 + 255) / 256));
  cudaError_t e =
      dtype == kF32
          ? launch_plain(sigmoid_gate_kernel<float>, grid, dim3(256), 0, stream, static_cast<float*>(o), ldo,
                     static_cast<const float*>(g), ldg, rows, c4)
          : launch_plain(sigmoid_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, static_cast<__nv_bfloat16*>(o), ldo,
                     static_cast<const __nv_bfloat16*>(g), ldg, rows, c4);
  return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}
