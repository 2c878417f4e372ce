// Latent attention of any size, in bf16 and fp32: the pieces around the latent cache and an attention kernel on the
// CUDA cores for what the tensor-core kernels (mla.cu, mla_tc.cu) do not take (fp32, latents wider than 512, rotated
// parts wider than 64).
//
//   mb_latent_post_down   after the fused down-projections of a layer: the query latent is RMS-normed; the key/value
//                         latent is RMS-normed and stored, with the rotated key part behind it, in the token's cache
//                         row. A layer that reads another layer's cache has no key/value columns and stores nothing.
//   mb_rotate_heads       rotates the first `dims` values of every head of a column block, in place
//   mb_latent_attention   absorbed attention over the paged rows [latent | rotated part], causal, with the options of
//                         MbAttnOptions (window, sink, output gate)
//
// Rows are padded: a cache row holds Rp >= R latent values and Dp >= rotated values, the rest is zero.
#include <cuda_runtime.h>

#include "../common/api.h"
#include "../common/head_gate.cuh"
#include "../common/launch.h"
#include "../common/scalar.cuh"

namespace mb {
namespace latent {

__device__ __forceinline__ float block_allsum(float v, float* scratch) {
  v = warp_allsum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < static_cast<int>(blockDim.x >> 5); ++i) t += scratch[i];
  return t;
}

// values i and j of a rotated pair number `pr`
__device__ __forceinline__ int2 pair_of(int pr, int dims, int interleaved) {
  return interleaved ? make_int2(2 * pr, 2 * pr + 1) : make_int2(pr, pr + dims / 2);
}

struct PostDown {
  int ld, q_rank, q_rank_pad, kv_off, R, Rp, rot_dim, Dp, dims, interleaved, ld_q, page_size, ld_cache;
  long long page_stride;
  float eps;
  const int32_t* positions;
  const float* cos_sin;      // [positions, dims]: dims / 2 cosines, then as many sines
  const int64_t* slots;
};

// RMS norm of one row by the CTA: dst[c] = src[c] / rms * gamma[c] for c < n, zeros up to n_pad. Rows whose pieces are
// aligned go through registers four values at a time (one read of `src`), others element by element.
template <typename T>
__device__ __forceinline__ void norm_row(const T* src, const T* gamma, T* dst, int n, int n_pad, float eps, bool vec, float* scratch) {
  const int tid = threadIdx.x;
  float ss = 0.f;
  if (vec) {                                 // n and n_pad are multiples of 4, n <= 4 * kVec * blockDim.x
    constexpr int kVec = 2;
    float4 x[kVec], g[kVec];
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
      const int c = (tid + i * blockDim.x) * 4;
      x[i] = c < n ? ld4(src + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      g[i] = c < n ? ld4(gamma + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
    }
    const float inv = 1.f / sqrtf(block_allsum(ss, scratch) / static_cast<float>(n) + eps);
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
      const int c = (tid + i * blockDim.x) * 4;
      if (c < n_pad) st4(dst + c, make_float4(x[i].x * inv * g[i].x, x[i].y * inv * g[i].y, x[i].z * inv * g[i].z, x[i].w * inv * g[i].w));
    }
    return;
  }
  for (int c = tid; c < n; c += blockDim.x) { const float v = ldf(src + c); ss += v * v; }
  const float inv = 1.f / sqrtf(block_allsum(ss, scratch) / static_cast<float>(n) + eps);
  for (int c = tid; c < n_pad; c += blockDim.x) stf(dst + c, c < n ? ldf(src + c) * inv * ldf(gamma + c) : 0.f);
}

__device__ __forceinline__ bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T>
__global__ void __launch_bounds__(256)
post_down_kernel(const PostDown p, const T* __restrict__ x, const T* __restrict__ gamma_q, const T* __restrict__ gamma_kv,
                 T* __restrict__ q_out, T* __restrict__ cache) {
  __shared__ float scratch[8];
  const int t = blockIdx.x, tid = threadIdx.x;
  const T* row = x + static_cast<size_t>(t) * p.ld;
  if (p.q_rank > 0) {
    T* o = q_out + static_cast<size_t>(t) * p.ld_q;
    norm_row(row, gamma_q, o, p.q_rank, p.q_rank_pad, p.eps,
             p.q_rank % 4 == 0 && p.q_rank_pad % 4 == 0 && p.q_rank_pad <= 8 * static_cast<int>(blockDim.x) && aligned16(row) &&
                 aligned16(gamma_q) && aligned16(o), scratch);
  }
  if (p.kv_off < 0) return;
  const int64_t slot = p.slots[t];
  if (slot < 0) return;                    // uniform over the CTA
  const T* kv = row + p.kv_off;
  T* dst = cache + (slot / p.page_size) * p.page_stride + (slot % p.page_size) * p.ld_cache;
  norm_row(kv, gamma_kv, dst, p.R, p.Rp, p.eps,
           p.R % 4 == 0 && p.Rp % 4 == 0 && p.Rp <= 8 * static_cast<int>(blockDim.x) && aligned16(kv) && aligned16(gamma_kv) &&
               aligned16(dst), scratch);
  const T* kr = kv + p.R;
  const float* cs = p.cos_sin + static_cast<size_t>(p.positions[t]) * p.dims;
  const int half = p.dims / 2;
  for (int i = tid; i < half; i += blockDim.x) {
    const int2 ij = pair_of(i, p.dims, p.interleaved);
    const float u = ldf(kr + ij.x), v = ldf(kr + ij.y), c = cs[i], s = cs[half + i];
    stf(dst + p.Rp + ij.x, u * c - v * s);
    stf(dst + p.Rp + ij.y, v * c + u * s);
  }
  for (int i = p.dims + tid; i < p.Dp; i += blockDim.x) stf(dst + p.Rp + i, i < p.rot_dim ? ldf(kr + i) : 0.f);
}

template <typename T>
__global__ void rotate_heads_kernel(T* __restrict__ x, int ld, int heads, int head_stride, int dims, int interleaved,
                                    const int32_t* __restrict__ positions, const float* __restrict__ cos_sin, int T_rows) {
  const int half = dims / 2;
  const long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= static_cast<long long>(T_rows) * heads * half) return;
  const int pr = static_cast<int>(i % half);
  const int h = static_cast<int>((i / half) % heads), t = static_cast<int>(i / half / heads);
  T* q = x + static_cast<size_t>(t) * ld + static_cast<size_t>(h) * head_stride;
  const float* cs = cos_sin + static_cast<size_t>(positions[t]) * dims;
  const int2 ij = pair_of(pr, dims, interleaved);
  const float u = ldf(q + ij.x), v = ldf(q + ij.y), c = cs[pr], s = cs[half + pr];
  stf(q + ij.x, u * c - v * s);
  stf(q + ij.y, v * c + u * s);
}

struct Attn {
  int ld_ql, ld_qr, hs_ql, hs_qr, ld_out, hs_out;   // token and head strides
  int B, bt_stride, page_size, ld_cache, Rp, Dp, n_heads;
  long long page_stride;
  const int32_t *block_table, *q_start, *q_len, *kv_len;
  const float* sink;
  HeadGate gate;
  int window;
  float scale;
};

constexpr int kWarps = 8;

// One CTA per (head, query token): eight warps share the keys, every lane keeps VPL columns of the running output.
template <typename T, int VPL>
__global__ void __launch_bounds__(kWarps * 32)
attention_kernel(const Attn p, const T* __restrict__ q_lat, const T* __restrict__ q_rope, const T* __restrict__ cache,
                 T* __restrict__ out) {
  extern __shared__ float sm[];                 // query row [Rp + Dp] | warp outputs [kWarps][Rp] | m, l
  const int head = blockIdx.x, t = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int LD = p.Rp + p.Dp;
  int lo = 0, hi = p.B - 1;                     // the last sequence that starts at or before t
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (p.q_start[mid] <= t) lo = mid; else hi = mid - 1;
  }
  const int off = t - p.q_start[lo];
  if (off >= p.q_len[lo]) return;               // a row of no sequence
  const int keys = p.kv_len[lo] - p.q_len[lo] + off + 1;
  const int first = keys > p.window ? keys - p.window : 0;
  const int32_t* bt = p.block_table + static_cast<size_t>(lo) * p.bt_stride;
  float* sq = sm;
  float* so = sm + LD;
  float* sml = so + kWarps * p.Rp;
  for (int c = tid; c < LD; c += blockDim.x)
    sq[c] = (c < p.Rp ? ldf(q_lat + static_cast<size_t>(t) * p.ld_ql + static_cast<size_t>(head) * p.hs_ql + c)
                      : ldf(q_rope + static_cast<size_t>(t) * p.ld_qr + static_cast<size_t>(head) * p.hs_qr + (c - p.Rp)));
  __syncthreads();
  float o[VPL];
#pragma unroll
  for (int i = 0; i < VPL; ++i) o[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int j = first + warp; j < keys; j += kWarps) {
    const T* row = cache + static_cast<size_t>(bt[j / p.page_size]) * p.page_stride +
                   static_cast<size_t>(j % p.page_size) * p.ld_cache;
    float k[VPL], s = 0.f;
#pragma unroll
    for (int i = 0; i < VPL; ++i) {
      const int c = lane + 32 * i;
      k[i] = c < p.Rp ? ldf(row + c) : 0.f;
      s = fmaf(k[i], c < p.Rp ? sq[c] : 0.f, s);
    }
    for (int c = p.Rp + lane; c < LD; c += 32) s = fmaf(ldf(row + c), sq[c], s);
    s = warp_allsum(s) * p.scale;
    const float mn = fmaxf(m, s);
    const float alpha = expf(m - mn), w = expf(s - mn);
    m = mn;
    l = l * alpha + w;
#pragma unroll
    for (int i = 0; i < VPL; ++i) o[i] = fmaf(w, k[i], o[i] * alpha);
  }
#pragma unroll
  for (int i = 0; i < VPL; ++i) {
    const int c = lane + 32 * i;
    if (c < p.Rp) so[warp * p.Rp + c] = o[i];
  }
  if (lane == 0) { sml[warp] = m; sml[kWarps + warp] = l; }
  __syncthreads();
  float M = p.sink ? p.sink[head] : -INFINITY;
#pragma unroll
  for (int i = 0; i < kWarps; ++i) M = fmaxf(M, sml[i]);
  float den = p.sink ? expf(p.sink[head] - M) : 0.f;
  float f[kWarps];
#pragma unroll
  for (int i = 0; i < kWarps; ++i) { f[i] = expf(sml[i] - M); den = fmaf(sml[kWarps + i], f[i], den); }
  const float inv = p.gate.of<T>(t, head) / den;
  T* dst = out + static_cast<size_t>(t) * p.ld_out + static_cast<size_t>(head) * p.hs_out;
  for (int c = tid; c < p.Rp; c += blockDim.x) {
    float v = 0.f;
#pragma unroll
    for (int i = 0; i < kWarps; ++i) v = fmaf(so[i * p.Rp + c], f[i], v);
    stf(dst + c, v * inv);
  }
}

template <typename T, int VPL>
static int launch_attn(const Attn& p, const void* ql, const void* qr, const void* cache, void* out, int T_rows,
                       cudaStream_t stream) {
  const size_t smem = (static_cast<size_t>(p.Rp + p.Dp) + static_cast<size_t>(kWarps) * p.Rp + 2 * kWarps) * sizeof(float);
  auto kern = attention_kernel<T, VPL>;
  static PerDeviceOnce configured;
  if (configured.needed()) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
      return MB_ERR_LAUNCH;
    configured.done();
  }
  if (smem > 200 * 1024) return MB_ERR_TOO_LARGE;
  // the grid's y dimension ends at 65535 rows; steps are far smaller
  if (T_rows > 65535) return MB_ERR_TOO_LARGE;
  return launch_plain(kern, dim3(p.n_heads, T_rows), dim3(kWarps * 32), smem, stream, p, static_cast<const T*>(ql),
                  static_cast<const T*>(qr), static_cast<const T*>(cache), static_cast<T*>(out)) == cudaSuccess
             ? MB_OK : MB_ERR_LAUNCH;
}

template <typename T>
static int dispatch_attn(const Attn& p, const void* ql, const void* qr, const void* cache, void* out, int T_rows,
                         cudaStream_t stream) {
  const int vpl = (p.Rp + 31) / 32;
  if (vpl <= 4) return launch_attn<T, 4>(p, ql, qr, cache, out, T_rows, stream);
  if (vpl <= 16) return launch_attn<T, 16>(p, ql, qr, cache, out, T_rows, stream);
  if (vpl <= 64) return launch_attn<T, 64>(p, ql, qr, cache, out, T_rows, stream);
  return MB_ERR_TOO_LARGE;
}

}  // namespace latent
}  // namespace mb

using namespace mb;

extern "C" int mb_latent_post_down(const void* x, int ld, int T, int q_rank, int q_rank_pad, const void* gamma_q,
                                   void* q_out, int ld_q, int kv_off, int R, int Rp, const void* gamma_kv, int rot_dim,
                                   int Dp, int dims, int interleaved, float eps, const int32_t* positions,
                                   const float* cos_sin, const int64_t* slots, void* cache, int page_size,
                                   long long page_stride, int ld_cache, int dtype, cudaStream_t stream) {
  if (T <= 0) return MB_OK;
  if (dims % 2 || dims > rot_dim || rot_dim > Dp || R > Rp || q_rank > q_rank_pad) return MB_ERR_SHAPE;
  latent::PostDown p = {ld, q_rank, q_rank_pad, kv_off, R, Rp, rot_dim, Dp, dims, interleaved, ld_q, page_size, ld_cache,
                        page_stride, eps, positions, cos_sin, slots};
  cudaError_t e;
  if (dtype == kF32)
    e = launch_plain(latent::post_down_kernel<float>, dim3(T), dim3(256), 0, stream, p, static_cast<const float*>(x),
                 static_cast<const float*>(gamma_q), static_cast<const float*>(gamma_kv), static_cast<float*>(q_out),
                 static_cast<float*>(cache));
  else
    e = launch_plain(latent::post_down_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, stream, p,
                 static_cast<const __nv_bfloat16*>(x), static_cast<const __nv_bfloat16*>(gamma_q),
                 static_cast<const __nv_bfloat16*>(gamma_kv), static_cast<__nv_bfloat16*>(q_out),
                 static_cast<__nv_bfloat16*>(cache));
  return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

extern "C" int mb_rotate_heads(void* x, int ld, int T, int heads, int head_stride, int dims, int interleaved,
                               const int32_t* positions, const float* cos_sin, int dtype, cudaStream_t stream) {
  if (T <= 0 || heads <= 0 || dims <= 0) return MB_OK;
  if (dims % 2 || dims > head_stride) return MB_ERR_SHAPE;
  const long long work = static_cast<long long>(T) * heads * (dims / 2);
  const dim3 grid(static_cast<unsigned>((work + 255) / 256));
  cudaError_t e = dtype == kF32
                      ? launch_plain(latent::rotate_heads_kernel<float>, grid, dim3(256), 0, stream, static_cast<float*>(x), ld,
                                 heads, head_stride, dims, interleaved, positions, cos_sin, T)
                      : launch_plain(latent::rotate_heads_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream,
                                 static_cast<__nv_bfloat16*>(x), ld, heads, head_stride, dims, interleaved, positions,
                                 cos_sin, T);
  return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

extern "C" int mb_latent_attention(const void* q_lat, int ld_ql, int hs_ql, const void* q_rope, int ld_qr, int hs_qr,
                                   void* out, int ld_out, int hs_out, const void* cache, long long page_stride,
                                   int ld_cache, int page_size, const int32_t* block_table, int bt_stride,
                                   const int32_t* q_start, const int32_t* q_len, const int32_t* kv_len, int T, int B,
                                   int n_heads, int Rp, int Dp, float scale, const MbAttnOptions* opt, int dtype,
                                   cudaStream_t stream) {
  if (T <= 0 || B <= 0) return MB_OK;
  if (ld_cache < Rp + Dp || n_heads <= 0) return MB_ERR_SHAPE;
  latent::Attn p = {ld_ql, ld_qr, hs_ql, hs_qr, ld_out, hs_out, B, bt_stride, page_size, ld_cache, Rp, Dp, n_heads,
                    page_stride, block_table, q_start, q_len, kv_len, opt ? opt->sink : nullptr, HeadGate(opt),
                    opt && opt->window > 0 ? opt->window : 0x7fffffff, scale};
  return dtype == kF32 ? latent::dispatch_attn<float>(p, q_lat, q_rope, cache, out, T, stream)
                       : latent::dispatch_attn<__nv_bfloat16>(p, q_lat, q_rope, cache, out, T, stream);
}
