// The seam between two branches of a decoder with an fp32 residual stream whose norms are elementwise: dynamic tanh,
//   T(y; alpha, w, b) = tanh(alpha * y) * w + b,
// before and after every branch, optionally with a token shift of what the next branch reads:
//
//   x'    = x + T(u; alpha_u, w_u, b_u)                    u: a branch output, and / or the weighted sum of expert outputs in
//                                                          expert order (identity experts give the row `self` back)
//   n1[t] = h[t]            or  h[t] + (h[t - 1] - h[t]) * shift,       h = T(x'; alpha_1, w1, b1)
//
// No value depends on another column, so there is no barrier and no reduction: a thread owns four columns and walks over a few
// tokens, the shifted row in registers. Ahead of its first token it computes the row before (from x, which a shifted seam
// therefore does not update in place: x' goes to a second buffer). Where a sequence continues, that row is in its state slot;
// the thread that owns a sequence's first token reads the slot and then stores the h of the sequence's last token in this step.
#include <cuda_runtime.h>

#include "../common/api.h"
#include "../common/launch.h"
#include "../common/scalar.cuh"

namespace mb {
namespace tanhseam {

// fp32 runs: the library's function. 16-bit runs: (1 - e) / (1 + e) with the fast exponential, a series below 1/4; relative error
// below 1e-6.
template <typename T>
__device__ __forceinline__ float tanh_of(float z) {
  if constexpr (sizeof(T) == 4) return tanhf(z);
  const float a = fabsf(z), e = __expf(-2.f * a), q = z * z;
  const float s = fmaf(q, fmaf(q, fmaf(q, fmaf(q, 62.f / 2835.f, -17.f / 315.f), 2.f / 15.f), -1.f / 3.f), 1.f) * a;
  return copysignf(a < 0.25f ? s : __fdividef(1.f - e, 1.f + e), z);
}

template <typename T>
__device__ __forceinline__ float4 affine_tanh(float4 y, float alpha, float4 w, float4 b) {
  return make_float4(fmaf(tanh_of<T>(alpha * y.x), w.x, b.x), fmaf(tanh_of<T>(alpha * y.y), w.y, b.y),
                     fmaf(tanh_of<T>(alpha * y.z), w.z, b.z), fmaf(tanh_of<T>(alpha * y.w), w.w, b.w));
}

// One pair of a token: the row of its expert's output (negative: none) and its weight.
struct __align__(8) Pair { int at; float w; };

// Many small CTAs per SM keep more rows in flight than several rows per thread would.
template <typename T, bool SHIFT, bool EXPERTS>
__global__ void __launch_bounds__(256, sizeof(T) == 4 ? 2 : EXPERTS ? 3 : SHIFT ? 6 : 8) tanh_seam_kernel(const MbTanhSeam p, int tile) {
  extern __shared__ Pair pairs[];                // EXPERTS: of the row before the tile, then of its rows
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
  const int tb = blockIdx.x * tile, te = min(tb + tile, p.n_rows), K = p.top_k;
  if (EXPERTS) {
    for (int i = threadIdx.x; i < (te - tb + 1) * K; i += blockDim.x) {
      const int t = tb - 1 + i / K;
      if (t < 0) continue;
      const size_t at = static_cast<size_t>(p.rows && t >= tb ? p.rows[t] : t) * K + i % K;
      pairs[i] = Pair{p.inverse[at], p.pair_w[at]};
    }
    __syncthreads();
  }
  if (c >= p.cols_pad) return;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  auto weight = [&](const void* w) { return w ? ld4(static_cast<const T*>(w) + c) : zero; };
  const float4 wu = weight(p.w_u), bu = weight(p.b_u), w1 = weight(p.w1), b1 = weight(p.b1);
  const float4 mix = SHIFT ? weight(p.shift) : zero;
  const bool update = p.a != nullptr || EXPERTS;
  // the stream and the branch of one row; `own`: its pairs, where they are staged
  auto load = [&](int row, const Pair* own, float4& x, float4& u) {
    x = u = zero;
    if (p.table) {
      const int64_t id = p.ids[row];
      if (id >= 0 && id < p.vocab) {
        x = ld4(static_cast<const T*>(p.table) + static_cast<size_t>(id) * p.ld_table + c);
        x.x *= p.scale; x.y *= p.scale; x.z *= p.scale; x.w *= p.scale;
      }
    } else {
      x = *reinterpret_cast<const float4*>(p.x + static_cast<size_t>(row) * p.ldx + c);
    }
    if (p.a) u = ld4(static_cast<const T*>(p.a) + static_cast<size_t>(row) * p.lda + c);
    if (EXPERTS) {
      // a pair without a row reads the token's own one: that of an identity expert, or any at weight zero
      const T* none = p.self ? static_cast<const T*>(p.self) + static_cast<size_t>(row) * p.ld_self + c : static_cast<const T*>(p.e) + c;
      const T* e = static_cast<const T*>(p.e) + c;
#pragma unroll 4
      for (int k = 0; k < K; ++k) {
        const Pair q = own ? own[k] : Pair{p.inverse[static_cast<size_t>(row) * K + k], p.pair_w[static_cast<size_t>(row) * K + k]};
        const float w = q.at >= 0 || p.self ? q.w : 0.f;
        const float4 y = ld4(q.at >= 0 ? e + static_cast<size_t>(q.at) * p.lde : none);
        u.x = fmaf(w, y.x, u.x); u.y = fmaf(w, y.y, u.y); u.z = fmaf(w, y.z, u.z); u.w = fmaf(w, y.w, u.w);
      }
    }
  };
  auto add = [&](float4& x, float4 u) {
    if (!update) return;
    const float4 y = affine_tanh<T>(u, p.alpha_u, wu, bu);
    x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
  };
  auto row_h = [&](int row, const Pair* own) {
    float4 x, u;
    load(row, own, x, u);
    add(x, u);
    return affine_tanh<T>(x, p.alpha_1, w1, b1);
  };
  int s = 0, first = 0, next = 0;                // SHIFT: the sequence of the current row, its first row and the one behind it
  float4 prev = zero, hx, hu;
  if (SHIFT) {
    load(max(tb - 1, 0), pairs + (tb > 0 ? 0 : K), hx, hu);
    s = tb;
    if (!p.one_token) {
      int lo = 0, hi = p.B - 1;                  // the last sequence that starts at or before the first row
      while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (p.q_start[mid] <= tb) lo = mid; else hi = mid - 1;
      }
      s = lo;
    }
    first = p.q_start[s];
    next = first + p.q_len[s];
  }
  for (int t = tb; t < te; ++t) {
    const int row = p.rows ? p.rows[t] : t;
    float4 x, u;
    load(row, pairs + (t - tb + 1) * K, x, u);
    if (SHIFT && t == tb && tb > first && tb < next) {
      add(hx, hu);
      prev = affine_tanh<T>(hx, p.alpha_1, w1, b1);
    }
    add(x, u);
    if (p.x_out) *reinterpret_cast<float4*>(p.x_out + static_cast<size_t>(row) * p.ldx + c) = x;
    if (!p.w1) continue;
    float4 h = affine_tanh<T>(x, p.alpha_1, w1, b1);
    if (SHIFT) {
      while (t >= next && s + 1 < p.B) { ++s; first = p.q_start[s]; next = first + p.q_len[s]; }
      if (t == first && t < next) {
        const int n = next - first, slot = p.state_idx[s];
        prev = zero;
        if (slot >= 0) {
          float* keep = p.prev + static_cast<size_t>(slot) * p.cols_pad + c;
          if (p.kv_len[s] > n) prev = *reinterpret_cast<const float4*>(keep);
          *reinterpret_cast<float4*>(keep) = n > 1 ? row_h(next - 1, nullptr) : h;
        }
      }
      const float4 d = make_float4(prev.x - h.x, prev.y - h.y, prev.z - h.z, prev.w - h.w);
      prev = h;
      h = make_float4(fmaf(d.x, mix.x, h.x), fmaf(d.y, mix.y, h.y), fmaf(d.z, mix.z, h.z), fmaf(d.w, mix.w, h.w));
    }
    st4(static_cast<T*>(p.n1) + static_cast<size_t>(t) * p.ld1 + c, h);
  }
}

template <typename T>
static int run(const MbTanhSeam& p, cudaStream_t stream) {
  // few rows: small CTAs over the columns of one row; many rows: each thread walks over some
  const int vec = p.cols_pad / 4, tile = p.n_rows <= 592 ? 1 : p.n_rows <= 4096 ? 4 : p.e ? 16 : 8;
  const int most = tile == 1 ? 128 : 256, threads = vec >= most ? most : (vec + 31) / 32 * 32;
  const dim3 grid((p.n_rows + tile - 1) / tile, (vec + threads - 1) / threads), block(threads);
  const size_t smem = p.e ? static_cast<size_t>(tile + 1) * p.top_k * sizeof(Pair) : 0;      // at most 4.3 KiB
  cudaError_t e;
  if (p.shift) e = p.e ? launch_plain(tanh_seam_kernel<T, true, true>, grid, block, smem, stream, p, tile)
                       : launch_plain(tanh_seam_kernel<T, true, false>, grid, block, smem, stream, p, tile);
  else e = p.e ? launch_plain(tanh_seam_kernel<T, false, true>, grid, block, smem, stream, p, tile)
               : launch_plain(tanh_seam_kernel<T, false, false>, grid, block, smem, stream, p, tile);
  return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

// ---- activations of a column range, in place
struct Xielu {
  float up, down;
  template <typename T>
  __device__ __forceinline__ float of(float z) const {
    const float m = fminf(z, 0.f);
    float g;                                     // exp(m) - 1 - m
    if constexpr (sizeof(T) == 4) g = expm1f(m) - m;
    else g = m > -0.25f ? m * m * fmaf(m, fmaf(m, fmaf(m, 1.f / 120.f, 1.f / 24.f), 1.f / 6.f), 0.5f) : __expf(m) - 1.f - m;
    return fmaf(0.5f, z, z > 0.f ? up * z * z : down * g);
  }
};
struct Tanh {
  template <typename T>
  __device__ __forceinline__ float of(float z) const { return tanh_of<T>(z); }
};

template <typename T, typename F>
__global__ void __launch_bounds__(256) activate_kernel(T* __restrict__ x, int ldx, int cols8, long long n8, F f) {
  const long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n8) return;
  T* q = x + (i / cols8) * ldx + (i % cols8) * 8;
  if constexpr (sizeof(T) == 2) {
    uint4 raw = *reinterpret_cast<const uint4*>(q);
    uint32_t* w = reinterpret_cast<uint32_t*>(&raw);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[k]));
      const __nv_bfloat162 b = __floats2bfloat162_rn(f.template of<T>(v.x), f.template of<T>(v.y));
      w[k] = *reinterpret_cast<const uint32_t*>(&b);
    }
    *reinterpret_cast<uint4*>(q) = raw;
  } else {
#pragma unroll
    for (int k = 0; k < 8; k += 4) {
      const float4 v = ld4(q + k);
      st4(q + k, make_float4(f.template of<T>(v.x), f.template of<T>(v.y), f.template of<T>(v.z), f.template of<T>(v.w)));
    }
  }
}

template <typename F>
static int activate(void* x, int ldx, int rows, int cols, F f, int dtype, cudaStream_t stream) {
  if (rows <= 0 || cols <= 0) return MB_OK;
  if (cols % 8 || ldx % 8) return MB_ERR_SHAPE;
  if (reinterpret_cast<uintptr_t>(x) & 15) return MB_ERR_ALIGN;
  const long long n8 = static_cast<long long>(rows) * (cols / 8);
  const dim3 grid(static_cast<unsigned>((n8 + 255) / 256));
  const cudaError_t e =
      dtype == kF32 ? launch_plain(activate_kernel<float, F>, grid, dim3(256), 0, stream, static_cast<float*>(x), ldx, cols / 8, n8, f)
                    : launch_plain(activate_kernel<__nv_bfloat16, F>, grid, dim3(256), 0, stream, static_cast<__nv_bfloat16*>(x), ldx,
                                   cols / 8, n8, f);
  return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

}  // namespace tanhseam
}  // namespace mb

using namespace mb;
using namespace mb::tanhseam;

extern "C" int mb_tanh_seam(const MbTanhSeam* p, int dtype, cudaStream_t stream) {
  if (p->n_rows <= 0) return MB_OK;
  if (p->cols_pad <= 0 || p->cols_pad % 4 || p->ldx % 4 || p->lda % 4 || p->lde % 4 || p->ld_self % 4 || p->ld1 % 4 || p->ld_table % 4 ||
      (p->e && (p->top_k <= 0 || p->top_k > 32)) || ((p->a || p->e) && !(p->w_u && p->b_u)) || (p->w1 && !(p->b1 && p->n1)))
    return MB_ERR_SHAPE;
  // a shifted seam reads rows that another thread has already updated, unless the update goes elsewhere
  if (p->shift && (!p->w1 || p->rows || !p->prev || p->B <= 0 || p->x_out == p->x)) return MB_ERR_SHAPE;
  return dtype == kF32 ? run<float>(*p, stream) : run<__nv_bfloat16>(*p, stream);
}

extern "C" int mb_tanh_cols(void* x, int ldx, int rows, int cols, int dtype, cudaStream_t stream) {
  return activate(x, ldx, rows, cols, Tanh{}, dtype, stream);
}

extern "C" int mb_xielu(void* x, int ldx, int rows, int cols, float up, float down, int dtype, cudaStream_t stream) {
  return activate(x, ldx, rows, cols, Xielu{up, down}, dtype, stream);
}
