// Lightning attention (linear attention with one constant decay per head) for ragged batches. Per head, with a state
// S [dim, vdim] in fp32:
//   S <- decay S + k v^T;   o = S^T q
//
//   lightning_scan_kernel   token by token on the CUDA cores, everything in fp32: decode steps, fp32 runs and heads wider
//                           than 128. Columns of S are independent, so a warp owns 4 NC of them: eight lanes share the rows
//                           of a column (RL4 float4 each, in registers). The state is read and written once per launch.
//   lightning_norm_kernel   the heads of a token, concatenated, RMS-normed together, scaled and gated
//
// State: [slot, head, column, row], rows padded to a size the scan is built for; `state_idx[s]` is the sequence's slot
// (-1: start from zero and keep nothing), read when the step continues a sequence (kv_len > q_len).
#include <cuda_runtime.h>

#include "../common/api.h"
#include "../common/launch.h"
#include "../common/scalar.cuh"

namespace mb {
namespace lightning {

template <typename T, int RL4, int NC, int MAXT>
__global__ void __launch_bounds__(MAXT) lightning_scan_kernel(const MbLightning p, int col_blocks, int chunk) {
  constexpr int DP = 32 * RL4;
  extern __shared__ __align__(16) float sm[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = lane & 7, cg = lane >> 3;
  const int V = p.vdim, cols = (blockDim.x >> 5) * 4 * NC;
  const int h = blockIdx.x / col_blocks, cbase = (blockIdx.x % col_blocks) * cols, s = blockIdx.y;
  const int t0 = p.q_start[s], n = p.q_len[s], slot = p.state_idx[s];
  if (n <= 0) return;
  const bool resume = slot >= 0 && p.kv_len[s] > n;
  const int lc = (warp * 4 + cg) * NC, col0 = cbase + lc;
  float* st = p.state + ((static_cast<size_t>(slot >= 0 ? slot : 0) * p.heads + h) * V + col0) * DP;
  float4 S[NC][RL4];
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int i = 0; i < RL4; ++i)
      S[c][i] = (resume && col0 + c < V) ? *reinterpret_cast<const float4*>(st + c * DP + (i * 8 + rg) * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
  const float g = p.decay[h];
  const int row_floats = 2 * DP + cols;
  const T* x = static_cast<const T*>(p.x);
  for (int c0 = 0; c0 < n; c0 += chunk) {
    const int m = min(chunk, n - c0);
    __syncthreads();
    for (int i = tid; i < m * row_floats; i += blockDim.x) {
      const int j = i / row_floats, c = i % row_floats;
      const T* row = x + static_cast<size_t>(t0 + c0 + j) * p.ldx;
      float v = 0.f;
      if (c < DP) { if (c < p.dim) v = ldf(row + p.q_off + h * p.dim + c); }
      else if (c < 2 * DP) { if (c - DP < p.dim) v = ldf(row + p.k_off + h * p.dim + c - DP); }
      else if (cbase + c - 2 * DP < V) v = ldf(row + p.v_off + h * V + cbase + c - 2 * DP);
      sm[i] = v;
    }
    __syncthreads();
#pragma unroll 2
    for (int j = 0; j < m; ++j) {
      const float* rp = sm + j * row_floats;
      float a[NC], v[NC];
#pragma unroll
      for (int c = 0; c < NC; ++c) { a[c] = 0.f; v[c] = rp[2 * DP + lc + c]; }
#pragma unroll
      for (int i = 0; i < RL4; ++i) {
        const int r = (i * 8 + rg) * 4;
        const float4 q = *reinterpret_cast<const float4*>(rp + r), k = *reinterpret_cast<const float4*>(rp + DP + r);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float4& e = S[c][i];
          e.x = fmaf(k.x, v[c], g * e.x); e.y = fmaf(k.y, v[c], g * e.y);
          e.z = fmaf(k.z, v[c], g * e.z); e.w = fmaf(k.w, v[c], g * e.w);
          a[c] = fmaf(e.x, q.x, a[c]); a[c] = fmaf(e.y, q.y, a[c]);
          a[c] = fmaf(e.z, q.z, a[c]); a[c] = fmaf(e.w, q.w, a[c]);
        }
      }
#pragma unroll
      for (int c = 0; c < NC; ++c) {
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) a[c] += __shfl_xor_sync(0xffffffffu, a[c], o);
        if (rg == c && col0 + c < V) stf(static_cast<T*>(p.o) + static_cast<size_t>(t0 + c0 + j) * p.ldo + h * V + col0 + c, a[c]);
      }
    }
  }
  if (slot >= 0) {
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int i = 0; i < RL4; ++i)
        if (col0 + c < V) *reinterpret_cast<float4*>(st + c * DP + (i * 8 + rg) * 4) = S[c][i];
  }
}

// o[t, :] = o / rms(o over the `n` true columns) * w * sigmoid(gate), in place; padding columns hold zeros
template <typename T>
__global__ void __launch_bounds__(1024) lightning_norm_kernel(T* __restrict__ o, int ldo, const T* __restrict__ gate, int ldg,
                                                              const T* __restrict__ w, int cols, int n, float eps) {
  __shared__ float part[32];
  const size_t t = blockIdx.x;
  T* row = o + t * ldo;
  const T* g = gate + t * ldg;
  float ss = 0.f;
  for (int c = threadIdx.x * 4; c < cols; c += blockDim.x * 4) {
    const float4 v = ld4(row + c);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  ss = warp_allsum(ss);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < static_cast<int>(blockDim.x >> 5); ++i) tot += part[i];
  const float inv = 1.f / sqrtf(tot / static_cast<float>(n) + eps);
  for (int c = threadIdx.x * 4; c < cols; c += blockDim.x * 4) {
    const float4 v = ld4(row + c), a = ld4(w + c), b = ld4(g + c);
    st4(row + c, make_float4(v.x * inv * a.x * sigmoidf(b.x), v.y * inv * a.y * sigmoidf(b.y), v.z * inv * a.z * sigmoidf(b.z),
                             v.w * inv * a.w * sigmoidf(b.w)));
  }
}

template <typename T, int RL4>
static int scan(const MbLightning& p, int num_sms, cudaStream_t stream) {
  constexpr int NC = RL4 <= 4 ? 2 : 1, MAXT = RL4 <= 8 ? 512 : 256, per_warp = 4 * NC;
  const int head_warps = (p.vdim + per_warp - 1) / per_warp;
  int warps = head_warps < MAXT / 32 ? head_warps : MAXT / 32;
  while (warps > 1 && static_cast<long long>(p.B) * p.heads * ((head_warps + warps - 1) / warps) < num_sms) warps = (warps + 1) / 2;
  const int cols = warps * per_warp, col_blocks = (p.vdim + cols - 1) / cols;
  const int per_token = (2 * 32 * RL4 + cols) * 4;
  int chunk = p.one_token ? 1 : 40 * 1024 / per_token;
  chunk = chunk > 16 ? 16 : chunk < 1 ? 1 : chunk;
  return launch_plain(lightning_scan_kernel<T, RL4, NC, MAXT>, dim3(p.heads * col_blocks, p.B), dim3(warps * 32),
                      static_cast<size_t>(chunk) * per_token, stream, p, col_blocks, chunk) == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

template <typename T>
static int run(const MbLightning& p, int num_sms, cudaStream_t stream) {
  switch (p.dim_pad / 32) {
    case 1: return scan<T, 1>(p, num_sms, stream);
    case 2: return scan<T, 2>(p, num_sms, stream);
    case 3: return scan<T, 3>(p, num_sms, stream);
    case 4: return scan<T, 4>(p, num_sms, stream);
    case 6: return scan<T, 6>(p, num_sms, stream);
    case 8: return scan<T, 8>(p, num_sms, stream);
    case 16: return scan<T, 16>(p, num_sms, stream);
    default: return MB_ERR_SHAPE;
  }
}

}  // namespace lightning
}  // namespace mb

using namespace mb;

extern "C" int mb_lightning(const MbLightning* p, int dtype, int num_sms, cudaStream_t stream) {
  if (p->T <= 0 || p->B <= 0) return MB_OK;
  if (p->heads <= 0 || p->dim <= 0 || p->vdim <= 0 || p->dim_pad != mb_delta_dim_pad(p->dim) || p->B > 65535) return MB_ERR_SHAPE;
  if (reinterpret_cast<uintptr_t>(p->state) & 15) return MB_ERR_ALIGN;
  return dtype == kF32 ? lightning::run<float>(*p, num_sms, stream) : lightning::run<__nv_bfloat16>(*p, num_sms, stream);
}

extern "C" int mb_lightning_norm(void* o, int ldo, const void* gate, int ldg, const void* w, int T, int cols, int n, float eps,
                                 int dtype, cudaStream_t stream) {
  if (T <= 0) return MB_OK;
  if (cols % 4 || ldo % 4 || ldg % 4 || n <= 0 || n > cols) return MB_ERR_SHAPE;
  const int most = T <= 296 ? 1024 : 256, nvec = cols / 4;
  const dim3 block(nvec >= most ? most : (nvec + 31) / 32 * 32);
  const cudaError_t e =
      dtype == kF32 ? launch_plain(lightning::lightning_norm_kernel<float>, dim3(T), block, 0, stream, static_cast<float*>(o), ldo,
                                   static_cast<const float*>(gate), ldg, static_cast<const float*>(w), cols, n, eps)
                    : launch_plain(lightning::lightning_norm_kernel<__nv_bfloat16>, dim3(T), block, 0, stream,
                                   static_cast<__nv_bfloat16*>(o), ldo, static_cast<const __nv_bfloat16*>(gate), ldg,
                                   static_cast<const __nv_bfloat16*>(w), cols, n, eps);
  return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}
