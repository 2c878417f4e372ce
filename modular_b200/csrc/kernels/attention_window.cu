// Softmax attention with a sliding window over the paged cache: what surrounds the tensor-core kernels
// (attention_tc.cu, attention_tma.cu), and a kernel on the CUDA cores for what those do not take (fp32, heads wider
// than 128, more than 16 query heads per key/value head, pages that are no multiple of 64 tokens).
//
//   mb_block_prep         everything between the stacked input projection of a parallel block and its branches, in one
//                         launch: queries rotated in place, keys rotated and stored in the cache with the values, silu on
//                         one column range and squared relu on another; or, with per-head norms, norms and rotation; or, with
//                         pairs half the rotated width apart, biases, rotation and store
//   mb_attention_plan     prompt tiles of a ragged step (sequence and first token of each), made on the device
//   mb_window_attention   causal attention of any head width, window and group size, optional sink score per head
//
// Cache: a token of page g, head h, offset o has its key at k_cache + g * page_stride + h * head_stride + o * hd.
#include <cuda_runtime.h>

#include "../common/api.h"
#include "../common/head_gate.cuh"
#include "../common/launch.h"
#include "../common/scalar.cuh"

namespace mb {
namespace winattn {

template <typename T>
struct Vec8 {
  float v[8];
  __device__ __forceinline__ void load(const T* p) {
    const float4 a = ld4(p), b = ld4(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
  __device__ __forceinline__ void store(T* p) const {
    st4(p, make_float4(v[0], v[1], v[2], v[3]));
    st4(p + 4, make_float4(v[4], v[5], v[6], v[7]));
  }
};
template <>
__device__ __forceinline__ void Vec8<__nv_bfloat16>::load(const __nv_bfloat16* p) {
  const uint4 r = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[i]));
    v[2 * i] = f.x; v[2 * i + 1] = f.y;
  }
}
template <>
__device__ __forceinline__ void Vec8<__nv_bfloat16>::store(__nv_bfloat16* p) const {
  uint32_t w[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    w[i] = *reinterpret_cast<const uint32_t*>(&b);
  }
  *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
}

// silu of an activation: fp32 runs take the accurate exponential, 16-bit runs (the result is rounded) the fast one
template <typename T>
__device__ __forceinline__ float act_silu(float z) {
  if constexpr (sizeof(T) == 4) return siluf(z);
  return __fdividef(z, 1.f + __expf(-z));
}

// values c0 .. c0 + 7 of a head at `cs` (one position's dims / 2 cosines, then as many sines); pairs are neighbours
template <typename T>
__device__ __forceinline__ void rotate8(Vec8<T>& x, const float* cs, int c0, int dims) {
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int pr = c0 / 2 + i;
    if (2 * pr >= dims) break;
    const float c = cs[pr], s = cs[dims / 2 + pr], u = x.v[2 * i], w = x.v[2 * i + 1];
    x.v[2 * i] = u * c - w * s;
    x.v[2 * i + 1] = w * c + u * s;
  }
}

template <typename T>
__global__ void __launch_bounds__(256) block_prep_kernel(const MbBlockPrep p) {
  const int t = blockIdx.x;
  int i = blockIdx.y * blockDim.x + threadIdx.x;           // 8-wide piece of this token's work
  T* row = static_cast<T*>(p.x) + static_cast<size_t>(t) * p.ldx;
  const int head8 = p.hd / 8, rot8 = (p.dims + 7) / 8;
  const float* cs = p.dims > 0 ? p.cos_sin + static_cast<size_t>(p.positions[t]) * p.dims : nullptr;
  Vec8<T> x;
  if (i < p.heads * rot8) {
    const int c = (i % rot8) * 8;
    T* q = row + p.q_off + (i / rot8) * p.hd + c;
    x.load(q);
    rotate8(x, cs, c, p.dims);
    x.store(q);
    return;
  }
  i -= p.heads * rot8;
  if (i < 2 * p.kv_heads * head8) {
    const bool is_v = i >= p.kv_heads * head8;
    if (is_v) i -= p.kv_heads * head8;
    const int h = i / head8, c = (i % head8) * 8;
    const int64_t slot = p.slots[t];
    if (slot < 0) return;
    x.load(row + (is_v ? p.v_off : p.k_off) + h * p.hd + c);
    if (!is_v && c < p.dims) rotate8(x, cs, c, p.dims);
    T* dst = static_cast<T*>(is_v ? p.v_cache : p.k_cache) + (slot / p.page_size) * p.page_stride + h * p.head_stride +
             static_cast<long long>(slot % p.page_size) * p.hd + c;
    x.store(dst);
    return;
  }
  i -= 2 * p.kv_heads * head8;
  if (i < p.silu_n / 8) {
    x.load(row + p.silu_off + i * 8);
#pragma unroll
    for (int k = 0; k < 8; ++k) x.v[k] = act_silu<T>(x.v[k]);
    x.store(row + p.silu_off + i * 8);
    return;
  }
  i -= p.silu_n / 8;
  if (i < p.relu2_n / 8) {
    x.load(row + p.relu2_off + i * 8);
#pragma unroll
    for (int k = 0; k < 8; ++k) { const float r = fmaxf(x.v[k], 0.f); x.v[k] = r * r; }
    x.store(row + p.relu2_off + i * 8);
  }
}

// The same for heads that are normed first, or whose pairs lie half the rotated width apart: a warp owns a head of a token.
template <typename T>
__global__ void __launch_bounds__(256) head_prep_kernel(const MbBlockPrep p) {
  extern __shared__ __align__(16) float rows[];            // one head per warp
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int u = blockIdx.y * (blockDim.x >> 5) + warp;
  if (u >= p.heads + 2 * p.kv_heads) return;
  T* row = static_cast<T*>(p.x) + static_cast<size_t>(t) * p.ldx;
  const bool is_q = u < p.heads, is_v = u >= p.heads + p.kv_heads;
  T *src = row + (is_q ? p.q_off + u * p.hd : (is_v ? p.v_off + (u - p.heads - p.kv_heads) * p.hd : p.k_off + (u - p.heads) * p.hd)),
    *dst = src;
  if (!is_q) {
    const int64_t slot = p.slots[t];
    if (slot < 0) return;
    const int h = is_v ? u - p.heads - p.kv_heads : u - p.heads;
    dst = static_cast<T*>(is_v ? p.v_cache : p.k_cache) + (slot / p.page_size) * p.page_stride + h * p.head_stride +
          static_cast<long long>(slot % p.page_size) * p.hd;
  }
  const float* bias = p.bias ? p.bias + (src - row) : nullptr;
  auto biased = [&](int c) {
    float4 x = ld4(src + c);
    if (bias) { const float4 b = *reinterpret_cast<const float4*>(bias + c); x.x += b.x; x.y += b.y; x.z += b.z; x.w += b.w; }
    return x;
  };
  if (is_v) {
    for (int c = lane * 4; c < p.hd; c += 128) st4(dst + c, biased(c));
    return;
  }
  float* s = rows + warp * p.hd;
  float ss = 0.f;
  for (int c = lane * 4; c < p.hd; c += 128) {
    const float4 x = biased(c);
    ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
    *reinterpret_cast<float4*>(s + c) = x;
  }
  const T* w = static_cast<const T*>(is_q ? p.q_norm : p.k_norm);
  if (w != nullptr) {
    const float inv = 1.f / sqrtf(warp_allsum(ss) / static_cast<float>(p.norm_dim) + p.eps);
    for (int c = lane * 4; c < p.hd; c += 128) {           // the columns this lane wrote
      const float4 x = *reinterpret_cast<const float4*>(s + c), g = ld4(w + c);
      *reinterpret_cast<float4*>(s + c) = make_float4(x.x * inv * g.x, x.y * inv * g.y, x.z * inv * g.z, x.w * inv * g.w);
    }
  }
  __syncwarp();
  const float* cs = p.dims > 0 ? p.cos_sin + static_cast<size_t>(p.positions[t]) * p.dims : nullptr;
  const int half = p.dims / 2;
  auto turned = [&](int c) {
    if (c >= p.dims) return s[c];
    const bool second = p.halves ? c >= half : (c & 1);
    const int pr = p.halves ? (second ? c - half : c) : c / 2;
    const int iu = p.halves ? pr : 2 * pr, iv = p.halves ? pr + half : 2 * pr + 1;
    return second ? s[iv] * cs[pr] + s[iu] * cs[half + pr] : s[iu] * cs[pr] - s[iv] * cs[half + pr];
  };
  for (int c = lane * 4; c < p.hd; c += 128) st4(dst + c, make_float4(turned(c), turned(c + 1), turned(c + 2), turned(c + 3)));
}

// Biases, rotation (pairs half the rotated width apart, that half a multiple of 8) and store, without norms: a thread owns eight
// pairs of a head, or eight columns that pass.
template <typename T>
__global__ void __launch_bounds__(256) pair_prep_kernel(const MbBlockPrep p, int q_items, int k_items, int v_items) {
  const int per = p.heads * q_items + p.kv_heads * (k_items + v_items);
  const long long id = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (id >= static_cast<long long>(p.T) * per) return;
  const int t = static_cast<int>(id / per), half = p.dims / 2, h8 = half / 8;
  int i = static_cast<int>(id % per), off, part;           // first column of the head in x, piece of the head
  T* row = static_cast<T*>(p.x) + static_cast<size_t>(t) * p.ldx;
  T* dst;
  bool turns = true;
  if (i < p.heads * q_items) {
    off = p.q_off + (i / q_items) * p.hd;
    part = i % q_items;
    dst = row + off;
  } else {
    i -= p.heads * q_items;
    const bool is_v = i >= p.kv_heads * k_items;
    if (is_v) i -= p.kv_heads * k_items;
    const int items = is_v ? v_items : k_items, h = i / items;
    const int64_t slot = p.slots[t];
    if (slot < 0) return;
    part = i % items;
    off = (is_v ? p.v_off : p.k_off) + h * p.hd;
    dst = static_cast<T*>(is_v ? p.v_cache : p.k_cache) + (slot / p.page_size) * p.page_stride + h * p.head_stride +
          static_cast<long long>(slot % p.page_size) * p.hd;
    turns = !is_v;
  }
  auto take = [&](Vec8<T>& x, int c) {
    x.load(row + off + c);
    if (!p.bias) return;
    const float4 a = *reinterpret_cast<const float4*>(p.bias + off + c), b = *reinterpret_cast<const float4*>(p.bias + off + c + 4);
    x.v[0] += a.x; x.v[1] += a.y; x.v[2] += a.z; x.v[3] += a.w; x.v[4] += b.x; x.v[5] += b.y; x.v[6] += b.z; x.v[7] += b.w;
  };
  Vec8<T> u;
  if (!turns || part >= h8) {
    const int c = turns ? p.dims + (part - h8) * 8 : part * 8;
    take(u, c);
    u.store(dst + c);
    return;
  }
  const int c = part * 8;
  Vec8<T> v;
  take(u, c);
  take(v, half + c);
  const float* cs = p.cos_sin + static_cast<size_t>(p.positions[t]) * p.dims + c;
  float co[8], si[8];
  *reinterpret_cast<float4*>(co) = *reinterpret_cast<const float4*>(cs); *reinterpret_cast<float4*>(co + 4) = *reinterpret_cast<const float4*>(cs + 4);
  *reinterpret_cast<float4*>(si) = *reinterpret_cast<const float4*>(cs + half); *reinterpret_cast<float4*>(si + 4) = *reinterpret_cast<const float4*>(cs + half + 4);
#pragma unroll
  for (int k = 0; k < 8; ++k) {
    const float a = u.v[k], b = v.v[k];
    u.v[k] = a * co[k] - b * si[k];
    v.v[k] = b * co[k] + a * si[k];
  }
  u.store(dst + c);
  v.store(dst + half + c);
}

constexpr int kPlanSeqs = 4096;

__global__ void __launch_bounds__(1024)
plan_kernel(const int32_t* __restrict__ q_len, int B, int tok, int n_tiles, int32_t* __restrict__ tile_seq, int32_t* __restrict__ tile_q0) {
  __shared__ int32_t first[kPlanSeqs + 1];
  __shared__ int32_t sums[32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int per = (B + 1023) / 1024, b0 = tid * per;
  int mine = 0;
  for (int b = b0; b < b0 + per && b < B; ++b) mine += (q_len[b] + tok - 1) / tok;
  int incl = mine;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int v = __shfl_up_sync(0xffffffffu, incl, o);
    if (lane >= o) incl += v;
  }
  if (lane == 31) sums[warp] = incl;
  __syncthreads();
  int base = 0;
  for (int w = 0; w < warp; ++w) base += sums[w];
  int run = base + incl - mine;
  for (int b = b0; b < b0 + per && b < B; ++b) {
    first[b] = run;
    run += (q_len[b] + tok - 1) / tok;
  }
  if (b0 < B && b0 + per >= B) first[B] = run;
  __syncthreads();
  const int total = first[B];
  for (int i = tid; i < n_tiles; i += blockDim.x) {
    int s = -1, q0 = 0;
    if (i < total) {
      int lo = 0, hi = B - 1;                     // the last sequence whose first tile is at or before i
      while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (first[mid] <= i) lo = mid; else hi = mid - 1;
      }
      s = lo;
      q0 = (i - first[lo]) * tok;
    }
    tile_seq[i] = s;
    tile_q0[i] = q0;
  }
}

struct Attn {
  int ldq, ldo, B, bt_stride, page_size, hd, G, window;
  long long page_stride, head_stride;
  const int32_t *block_table, *q_start, *q_len, *kv_len;
  const float* sink;
  HeadGate gate;
  float scale;
};

constexpr int kWarps = 8;

// One CTA per (query token, head): eight warps share the keys, every lane keeps VPL columns of the running output.
template <typename T, int VPL>
__global__ void __launch_bounds__(kWarps * 32)
attention_kernel(const Attn p, const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache, T* __restrict__ out) {
  extern __shared__ float sm[];                 // query row [hd] | warp outputs [kWarps][hd] | m, l
  const int t = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int lo = 0, hi = p.B - 1;                     // the last sequence that starts at or before t
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (p.q_start[mid] <= t) lo = mid; else hi = mid - 1;
  }
  const int off = t - p.q_start[lo];
  if (off < 0 || off >= p.q_len[lo]) return;    // a row of no sequence
  const int pos = p.kv_len[lo] - p.q_len[lo] + off;
  const int first = pos - p.window + 1 > 0 ? pos - p.window + 1 : 0;
  const int32_t* bt = p.block_table + static_cast<size_t>(lo) * p.bt_stride;
  float *so = sm + p.hd, *sml = so + kWarps * p.hd;
  for (int c = tid; c < p.hd; c += blockDim.x) sm[c] = ldf(q + static_cast<size_t>(t) * p.ldq + static_cast<size_t>(head) * p.hd + c);
  __syncthreads();
  const long long hoff = (head / p.G) * p.head_stride;
  float o[VPL], qv[VPL];
#pragma unroll
  for (int i = 0; i < VPL; ++i) { const int c = lane + 32 * i; o[i] = 0.f; qv[i] = c < p.hd ? sm[c] : 0.f; }
  float m = -INFINITY, l = 0.f;
  for (int j = first + warp; j <= pos; j += kWarps) {
    const long long e = bt[j / p.page_size] * p.page_stride + hoff + static_cast<long long>(j % p.page_size) * p.hd;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < VPL; ++i) { const int c = lane + 32 * i; if (c < p.hd) s = fmaf(ldf(k_cache + e + c), qv[i], s); }
    s = warp_allsum(s) * p.scale;
    const float mn = fmaxf(m, s);
    const float alpha = expf(m - mn), w = expf(s - mn);
    m = mn;
    l = l * alpha + w;
#pragma unroll
    for (int i = 0; i < VPL; ++i) { const int c = lane + 32 * i; if (c < p.hd) o[i] = fmaf(w, ldf(v_cache + e + c), o[i] * alpha); }
  }
#pragma unroll
  for (int i = 0; i < VPL; ++i) { const int c = lane + 32 * i; if (c < p.hd) so[warp * p.hd + c] = o[i]; }
  if (lane == 0) { sml[warp] = m; sml[kWarps + warp] = l; }
  __syncthreads();
  float M = p.sink ? p.sink[head] : -INFINITY;
#pragma unroll
  for (int i = 0; i < kWarps; ++i) M = fmaxf(M, sml[i]);
  float den = p.sink ? expf(p.sink[head] - M) : 0.f, f[kWarps];
#pragma unroll
  for (int i = 0; i < kWarps; ++i) { f[i] = expf(sml[i] - M); den = fmaf(sml[kWarps + i], f[i], den); }
  const float inv = p.gate.of<T>(t, head) / den;
  T* dst = out + static_cast<size_t>(t) * p.ldo + static_cast<size_t>(head) * p.hd;
  for (int c = tid; c < p.hd; c += blockDim.x) {
    float v = 0.f;
#pragma unroll
    for (int i = 0; i < kWarps; ++i) v = fmaf(so[i * p.hd + c], f[i], v);
    stf(dst + c, v * inv);
  }
}

template <typename T, int VPL>
static int launch_attn(const Attn& p, const void* q, const void* k, const void* v, void* out, int T_rows, int heads, cudaStream_t stream) {
  const size_t smem = (static_cast<size_t>(1 + kWarps) * p.hd + 2 * kWarps) * sizeof(float);   // at most 37 KiB
  return launch_plain(attention_kernel<T, VPL>, dim3(T_rows, heads), dim3(kWarps * 32), smem, stream, p, static_cast<const T*>(q),
                      static_cast<const T*>(k), static_cast<const T*>(v), static_cast<T*>(out)) == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

template <typename T>
static int dispatch(const Attn& p, const void* q, const void* k, const void* v, void* out, int T_rows, int heads, cudaStream_t stream) {
  if (p.hd <= 128) return launch_attn<T, 4>(p, q, k, v, out, T_rows, heads, stream);
  if (p.hd <= 256) return launch_attn<T, 8>(p, q, k, v, out, T_rows, heads, stream);
  if (p.hd <= 512) return launch_attn<T, 16>(p, q, k, v, out, T_rows, heads, stream);
  if (p.hd <= 1024) return launch_attn<T, 32>(p, q, k, v, out, T_rows, heads, stream);
  return MB_ERR_TOO_LARGE;
}

}  // namespace winattn
}  // namespace mb

using namespace mb;

extern "C" int mb_block_prep(const MbBlockPrep* p, int dtype, cudaStream_t stream) {
  if (p->T <= 0) return MB_OK;
  if (p->hd % 8 || p->dims % 2 || p->dims > p->hd || p->ldx % 8 || p->q_off % 8 || p->k_off % 8 || p->v_off % 8 ||
      p->silu_off % 8 || p->silu_n % 8 || p->relu2_off % 8 || p->relu2_n % 8)
    return MB_ERR_SHAPE;
  if ((reinterpret_cast<uintptr_t>(p->x) | reinterpret_cast<uintptr_t>(p->k_cache) | reinterpret_cast<uintptr_t>(p->v_cache)) & 15)
    return MB_ERR_ALIGN;
  if (p->bias && (!p->halves || (reinterpret_cast<uintptr_t>(p->bias) & 15))) return MB_ERR_SHAPE;
  if (!p->q_norm && !p->k_norm && p->halves && p->dims % 16 == 0 && !p->silu_n && !p->relu2_n &&
      (reinterpret_cast<uintptr_t>(p->cos_sin) & 15) == 0) {
    const int rot = p->dims / 16, rest = (p->hd - p->dims) / 8, q = rot + (p->bias ? rest : 0);
    const long long n = static_cast<long long>(p->T) * (p->heads * q + p->kv_heads * (rot + rest + p->hd / 8));
    if (n == 0) return MB_OK;
    const dim3 g(static_cast<unsigned>((n + 255) / 256));
    const cudaError_t e = dtype == kF32 ? launch_plain(winattn::pair_prep_kernel<float>, g, dim3(256), 0, stream, *p, q, rot + rest, p->hd / 8)
                                        : launch_plain(winattn::pair_prep_kernel<__nv_bfloat16>, g, dim3(256), 0, stream, *p, q, rot + rest, p->hd / 8);
    return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
  }
  if (p->q_norm || p->k_norm || p->halves) {
    if (p->silu_n || p->relu2_n || p->norm_dim <= 0 || p->norm_dim > p->hd || p->hd > 1024) return MB_ERR_SHAPE;
    const dim3 g(p->T, (p->heads + 2 * p->kv_heads + 7) / 8);
    const size_t smem = static_cast<size_t>(8) * p->hd * sizeof(float);      // at most 32 KiB
    const cudaError_t e = dtype == kF32 ? launch_plain(winattn::head_prep_kernel<float>, g, dim3(256), smem, stream, *p)
                                        : launch_plain(winattn::head_prep_kernel<__nv_bfloat16>, g, dim3(256), smem, stream, *p);
    return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
  }
  const long long work = static_cast<long long>(p->heads) * ((p->dims + 7) / 8) + 2ll * p->kv_heads * (p->hd / 8) + p->silu_n / 8 +
                         p->relu2_n / 8;
  const long long blocks = (work + 255) / 256;
  if (blocks == 0) return MB_OK;
  if (blocks > 65535) return MB_ERR_TOO_LARGE;
  const dim3 grid(p->T, static_cast<unsigned>(blocks));
  const cudaError_t e = dtype == kF32 ? launch_plain(winattn::block_prep_kernel<float>, grid, dim3(256), 0, stream, *p)
                                      : launch_plain(winattn::block_prep_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, *p);
  return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

extern "C" int mb_attention_plan(const int32_t* q_len, int B, int tok_per_tile, int n_tiles, int32_t* tile_seq, int32_t* tile_q0,
                                 cudaStream_t stream) {
  if (n_tiles <= 0 || B <= 0) return MB_OK;
  if (tok_per_tile <= 0) return MB_ERR_SHAPE;
  if (B > winattn::kPlanSeqs) return MB_ERR_TOO_LARGE;
  return launch_plain(winattn::plan_kernel, dim3(1), dim3(1024), 0, stream, q_len, B, tok_per_tile, n_tiles, tile_seq, tile_q0) ==
                 cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

extern "C" int mb_window_attention(const void* q, int ldq, void* out, int ldo, const void* k_cache, const void* v_cache,
                                   long long page_stride, long long head_stride, int page_size, const int32_t* block_table,
                                   int bt_stride, const int32_t* q_start, const int32_t* q_len, const int32_t* kv_len, int T, int B,
                                   int n_q, int n_kv, int hd, float scale, const MbAttnOptions* opt, int dtype,
                                   cudaStream_t stream) {
  if (T <= 0 || B <= 0) return MB_OK;
  if (n_kv <= 0 || n_q % n_kv || n_q > 65535 || hd <= 0) return MB_ERR_SHAPE;
  winattn::Attn p = {ldq, ldo, B, bt_stride, page_size, hd, n_q / n_kv, opt && opt->window > 0 ? opt->window : 0x7fffffff, page_stride, head_stride,
                     block_table, q_start, q_len, kv_len, opt ? opt->sink : nullptr, HeadGate(opt), scale};
  return dtype == kF32 ? winattn::dispatch<float>(p, q, k_cache, v_cache, out, T, n_q, stream)
                       : winattn::dispatch<__nv_bfloat16>(p, q, k_cache, v_cache, out, T, n_q, stream);
}
