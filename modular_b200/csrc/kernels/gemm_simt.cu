// fp32 products on the CUDA cores: Y = X . W^T with fp32 operands and fp32 accumulation, for serving a model in true
// 32-bit arithmetic. Three shapes share the kernel:
//   plain     Y[m, n] = sum_k X[m, k] W[n, k] (+ R[m, n])
//   batched   Y[m, z * y_off + n] = sum_k X[m, z * x_off + k] W[z, n, k]        (per-head products)
//   grouped   rows [offsets[z], offsets[z + 1]) of X times W[z]                  (experts)
// 64 x 64 output tile, 16-deep K steps through shared memory, 4 x 4 outputs per thread. Any M, N, K.
#include <cuda_runtime.h>

#include "../common/api.h"
#include "../common/launch.h"

namespace mb {
namespace simt {

constexpr int kBM = 64, kBN = 64, kBK = 16, kPad = 4;

struct Params {
  const float* x;
  const float* w;
  const float* r;
  float* y;
  int M, N, K, ldx, ldw, ldy, ldr, x_off, y_off;
  long long w_stride;
  const int32_t* offsets;
};

__global__ void __launch_bounds__(256) gemm_simt_kernel(const Params p) {
  __shared__ __align__(16) float sx[kBK][kBM + kPad];
  __shared__ __align__(16) float sw[kBK][kBN + kPad];
  const int z = blockIdx.z;
  int m_begin = 0, m_end = p.M;
  if (p.offsets) { m_begin = p.offsets[z]; m_end = p.offsets[z + 1]; }
  const int m0 = m_begin + blockIdx.y * kBM, n0 = blockIdx.x * kBN;
  if (m0 >= m_end) return;
  const float* X = p.x + static_cast<long long>(z) * p.x_off;
  const float* W = p.w + static_cast<long long>(z) * p.w_stride;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += kBK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = tid + i * 256, row = idx >> 4, kk = idx & 15;
      const int k = k0 + kk;
      sx[kk][row] = (m0 + row < m_end && k < p.K) ? X[static_cast<long long>(m0 + row) * p.ldx + k] : 0.f;
      sw[kk][row] = (n0 + row < p.N && k < p.K) ? W[static_cast<long long>(n0 + row) * p.ldw + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kBK; ++kk) {
      const float4 a = *reinterpret_cast<const float4*>(&sx[kk][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&sw[kk][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= m_end) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= p.N) continue;
      float v = acc[i][j];
      if (p.r) v += p.r[static_cast<long long>(m) * p.ldr + n];
      p.y[static_cast<long long>(m) * p.ldy + static_cast<long long>(z) * p.y_off + n] = v;
    }
  }
}

// out[r, i] = silu(gu[r, i]) * gu[r, inter + i]
__global__ void silu_mul_f32_kernel(const float* __restrict__ gu, float* __restrict__ out, size_t n, int inter) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const size_t r = i / inter, c = i % inter;
  const float g = gu[r * 2 * inter + c];
  out[i] = g / (1.f + expf(-g)) * gu[r * 2 * inter + inter + c];
}

static int launch(const Params& p, int m_rows, int batches, cudaStream_t stream) {
  const dim3 grid((p.N + kBN - 1) / kBN, (m_rows + kBM - 1) / kBM, batches);
  if (grid.y > 65535 || grid.z > 65535) return MB_ERR_TOO_LARGE;
  return launch_plain(gemm_simt_kernel, grid, dim3(256), 0, stream, p) == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

}  // namespace simt
}  // namespace mb

using namespace mb;

extern "C" int mb_gemm_f32(const float* x, const float* w, float* y, const float* r, int M, int N, int K, int ldx,
                           int ldw, int ldy, int ldr, cudaStream_t stream) {
  if (M <= 0 || N <= 0) return MB_OK;
  simt::Params p = {x, w, r, y, M, N, K, ldx, ldw, ldy, ldr, 0, 0, 0, nullptr};
  return simt::launch(p, M, 1, stream);
}

extern "C" int mb_batched_gemm_f32(const float* x, const float* w, float* y, int B, int M, int N, int K, int ldx,
                                   int x_off, int ldy, int y_off, cudaStream_t stream) {
  if (B <= 0 || M <= 0 || N <= 0) return MB_OK;
  simt::Params p = {x, w, nullptr, y, M, N, K, ldx, K, ldy, 0, x_off, y_off, static_cast<long long>(N) * K, nullptr};
  return simt::launch(p, M, B, stream);
}

extern "C" int mb_grouped_gemm_f32(const float* x, const float* w, float* y, const int32_t* offsets, int E, int max_rows,
                                   int N, int K, cudaStream_t stream) {
  if (E <= 0 || max_rows <= 0 || N <= 0) return MB_OK;
  simt::Params p = {x, w, nullptr, y, max_rows, N, K, K, K, N, 0, 0, 0, static_cast<long long>(N) * K, offsets};
  return simt::launch(p, max_rows, E, stream);
}

extern "C" int mb_silu_mul_f32(const float* gu, float* out, int rows, int inter, cudaStream_t stream) {
  if (rows <= 0 || inter <= 0) return MB_OK;
  const size_t n = static_cast<size_t>(rows) * inter;
  return launch_plain(simt::silu_mul_f32_kernel, dim3(static_cast<unsigned>((n + 255) / 256)), dim3(256), 0, stream, gu, out,
                  n, inter) == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}
