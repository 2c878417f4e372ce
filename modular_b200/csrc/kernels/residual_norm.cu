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
// Also here: tanh-GELU in place and the sigmoid output gate of an attention layer.
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
  return launch_plain(residual_norm_kernel<T>, dim3(q.n_rows), dim3(threads), static_cast<size_t>(p.cols_pad) * 4, stream, p) ==
                 cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

template <typename T>
__global__ void gelu_tanh_kernel(T* __restrict__ x, size_t n4) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n4) return;
  const float4 v = ld4(x + i * 4);
  auto f = [](float z) { return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); };
  st4(x + i * 4, make_float4(f(v.x), f(v.y), f(v.z), f(v.w)));
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
      q->ld1 % 4 || q->ld2 % 4 || q->ld_table % 4)
    return MB_ERR_SHAPE;
  if (q->cols_pad > 12288) return MB_ERR_TOO_LARGE;
  return dtype == kF32 ? run<float>(*q, stream) : run<__nv_bfloat16>(*q, stream);
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
