// Lightning attention (linear attention with one constant decay per head) for ragged batches. Per head, with a state
// S [dim, vdim] in fp32:
//   S <- decay S + k v^T;   o = S^T q
//
//   lightning_scan_kernel   token by token on the CUDA cores, everything in fp32: decode steps, fp32 runs and heads wider
//                           than 128. Columns of S are independent, so a warp owns 4 NC of them: eight lanes share the rows
//                           of a column (RL4 float4 each, in registers). The state is read and written once per launch.
//   lightning_chunk_kernel  bf16 prompts of heads up to 128 wide, 64 tokens at a time on the tensor cores. With powers of
//                           the decay g, rows i, j of a chunk and the state S before it:
//                             o_i = g^(i+1) S^T q_i + sum_{j <= i} g^(i-j) (q_i . k_j) v_j
//                             S'  = g^m S + sum_j k_j (g^(m-1-j) v_j)^T                     (m tokens in the chunk)
//                           q, k and v are 16-bit activations; everything made from them (S, the weighted products
//                           q . k, the decayed values) is fp32 and enters a product as the sum of two bf16 numbers, so no
//                           term is rounded to 16 bits. S^T stays in the accumulator fragments of the warp that owns its
//                           16 columns, which are also the B fragments of S^T q: the state never passes through shared
//                           memory, and a chunk needs two barriers. That dependency from chunk to chunk is why this runs
//                           on mma.sync: with the state in TMEM every chunk would move it to shared memory and back.
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

constexpr int kChunk = 64, kNV = 64, kWarps = 4, kThreads = kWarps * 32;
constexpr int kLdV = kNV + 8, kLdP = kChunk + 8;     // padded rows: conflict-free ldmatrix

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)) : "memory");
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// x, y as the sums of two bf16 numbers each
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

// Products of 16 queries (rows 16 W ..) with the keys at or before them, decayed, into sP as hi and lo parts.
template <int W, int DK>
__device__ __forceinline__ void chunk_products(const __nv_bfloat16* sQ, const __nv_bfloat16* sK, __nv_bfloat16* sP, const float* pw, int lane) {
  constexpr int LDK = DK + 8;
  const int mi = lane >> 3, r8 = lane & 7, row4 = lane >> 2, col2 = 2 * (lane & 3);
  float sc[2 * (W + 1)][4];
#pragma unroll
  for (int i = 0; i < 2 * (W + 1); ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
#pragma unroll
  for (int kb = 0; kb < DK / 16; ++kb) {
    uint32_t a[4];
    ldsm4(a, sQ + (W * 16 + (lane & 15)) * LDK + kb * 16 + (lane >> 4) * 8);
#pragma unroll
    for (int np = 0; np <= W; ++np) {
      uint32_t b[4];
      ldsm4(b, sK + (np * 16 + (mi >> 1) * 8 + r8) * LDK + kb * 16 + (mi & 1) * 8);
      mma(sc[2 * np], a, b[0], b[1]);
      mma(sc[2 * np + 1], a, b[2], b[3]);
    }
  }
#pragma unroll
  for (int nt = 0; nt < 2 * (W + 1); ++nt)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = W * 16 + row4 + 8 * e, d = i - (nt * 8 + col2);            // distance to the first of two keys
      const float a0 = d >= 0 ? sc[nt][2 * e] * pw[d] : 0.f, a1 = d >= 1 ? sc[nt][2 * e + 1] * pw[d - 1] : 0.f;
      uint32_t hi, lo;
      split2(a0, a1, hi, lo);
      *reinterpret_cast<uint32_t*>(sP + i * kLdP + nt * 8 + col2) = hi;
      *reinterpret_cast<uint32_t*>(sP + (kChunk + i) * kLdP + nt * 8 + col2) = lo;
    }
}

// One CTA walks the chunks of one (sequence, head, 64 value columns). DK: key width padded to a multiple of 32.
template <int DK>
__global__ void __launch_bounds__(kThreads, 2) lightning_chunk_kernel(const MbLightning p, int col_blocks) {
  typedef __nv_bfloat16 bf16;
  constexpr int LDK = DK + 8, KB = DK / 16, kStage = kChunk * (2 * LDK + kLdV);
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* stages = reinterpret_cast<bf16*>(smem_raw);
  bf16* sP = stages + 2 * kStage;                    // [hi | lo][chunk][kLdP]: weighted products q . k
  __shared__ float pw[kChunk + 1];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mi = lane >> 3, r8 = lane & 7, row4 = lane >> 2, col2 = 2 * (lane & 3);
  const int h = blockIdx.x / col_blocks, v0 = (blockIdx.x % col_blocks) * kNV, s = blockIdx.y, V = p.vdim;
  const int t0 = p.q_start[s], n = p.q_len[s], slot = p.state_idx[s];
  if (n <= 0) return;
  const bool resume = slot >= 0 && p.kv_len[s] > n;
  for (int i = tid; i <= kChunk; i += kThreads) pw[i] = p.decay_pow[h * (kChunk + 1) + i];
  const bf16* x = static_cast<const bf16*>(p.x) + static_cast<size_t>(t0) * p.ldx;
  auto fetch = [&](int c0, bf16* dst) {              // rows beyond the sequence and columns beyond the head become zero
    constexpr int CH = DK / 8;
    for (int i = tid; i < kChunk * CH; i += kThreads) {
      const int j = i / CH, c = (i % CH) * 8;
      const bool ok = c0 + j < n && c < p.dim;
      const bf16* src = x + (ok ? static_cast<size_t>(c0 + j) * p.ldx + h * p.dim + c : 0);
      cp_async16(dst + j * LDK + c, src + (ok ? p.q_off : 0), ok);
      cp_async16(dst + (kChunk + j) * LDK + c, src + (ok ? p.k_off : 0), ok);
    }
    bf16* dv = dst + 2 * kChunk * LDK;
    for (int i = tid; i < kChunk * (kNV / 8); i += kThreads) {
      const int j = i / (kNV / 8), c = (i % (kNV / 8)) * 8;
      const bool ok = c0 + j < n && v0 + c < V;
      cp_async16(dv + j * kLdV + c, x + (ok ? static_cast<size_t>(c0 + j) * p.ldx + p.v_off + h * V + v0 + c : 0), ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, stages);
  // S^T: 16 value columns of this warp as accumulator tiles of 8 keys: [0], [1] value row4, [2], [3] value row4 + 8
  float S[2 * KB][4];
  float* st = p.state + (static_cast<size_t>(slot >= 0 ? slot : 0) * p.heads + h) * V * DK;
  const int vr = v0 + warp * 16 + row4;
#pragma unroll
  for (int t = 0; t < 2 * KB; ++t)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float2 f = make_float2(0.f, 0.f);
      if (resume && vr + 8 * e < V) f = *reinterpret_cast<const float2*>(st + static_cast<size_t>(vr + 8 * e) * DK + 8 * t + col2);
      S[t][2 * e] = f.x; S[t][2 * e + 1] = f.y;
    }
  bool have_state = resume;
  for (int c0 = 0, it = 0; c0 < n; c0 += kChunk, ++it) {
    const int m = min(kChunk, n - c0);
    const bf16 *sQ = stages + (it & 1) * kStage, *sK = sQ + kChunk * LDK, *sV = sK + kChunk * LDK;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                 // this chunk is in; the last one is done with its stage and with sP
    if (c0 + kChunk < n) fetch(c0 + kChunk, stages + ((it + 1) & 1) * kStage);
    // straight-line code from here on: rows beyond the end of the sequence are zeros and cost what full ones cost
    switch (warp) {
      case 0: chunk_products<0, DK>(sQ, sK, sP, pw, lane); break;
      case 1: chunk_products<1, DK>(sQ, sK, sP, pw, lane); break;
      case 2: chunk_products<2, DK>(sQ, sK, sP, pw, lane); break;
      default: chunk_products<3, DK>(sQ, sK, sP, pw, lane); break;
    }
    // what the state before the chunk contributes, for all queries and this warp's 16 value columns
    float o[4][2][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;
    if (have_state) {
#pragma unroll
      for (int kb = 0; kb < KB; ++kb) {
        uint32_t hi[2][2], lo[2][2];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e) split2(S[2 * kb + e][2 * j], S[2 * kb + e][2 * j + 1], hi[j][e], lo[j][e]);
        uint32_t a[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) ldsm4(a[i], sQ + (i * 16 + (lane & 15)) * LDK + kb * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int i = 0; i < 4; ++i) { mma(o[i][0], a[i], hi[0][0], hi[0][1]); mma(o[i][1], a[i], hi[1][0], hi[1][1]); }
#pragma unroll
        for (int i = 0; i < 4; ++i) { mma(o[i][0], a[i], lo[0][0], lo[0][1]); mma(o[i][1], a[i], lo[1][0], lo[1][1]); }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float f0 = pw[i * 16 + row4 + 1], f1 = pw[i * 16 + row4 + 9];
#pragma unroll
        for (int j = 0; j < 2; ++j) { o[i][j][0] *= f0; o[i][j][1] *= f0; o[i][j][2] *= f1; o[i][j][3] *= f1; }
      }
    }
    __syncthreads();                                 // the products of every warp are in sP
#pragma unroll
    for (int kb = 0; kb < 4; ++kb) {
      uint32_t b[4];
      ldsm4_t(b, sV + (kb * 16 + (mi & 1) * 8 + r8) * kLdV + warp * 16 + (mi >> 1) * 8);
#pragma unroll
      for (int half = 0; half < 2; ++half) {
#pragma unroll
        for (int i = kb; i < 4; ++i) {
          uint32_t a[4];
          ldsm4(a, sP + (half * kChunk + i * 16 + (lane & 15)) * kLdP + kb * 16 + (lane >> 4) * 8);
          mma(o[i][0], a, b[0], b[1]);
          mma(o[i][1], a, b[2], b[3]);
        }
      }
    }
    bf16* out = static_cast<bf16*>(p.o) + static_cast<size_t>(t0 + c0) * p.ldo + h * V;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = i * 16 + row4 + 8 * e;
        if (r >= m) continue;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int c = v0 + warp * 16 + j * 8 + col2;
          if (c < V) *reinterpret_cast<__nv_bfloat162*>(out + static_cast<size_t>(r) * p.ldo + c) = __floats2bfloat162_rn(o[i][j][2 * e], o[i][j][2 * e + 1]);
        }
      }
    // the state after the chunk
    if (have_state) {
      const float f = pw[m];
#pragma unroll
      for (int t = 0; t < 2 * KB; ++t) { S[t][0] *= f; S[t][1] *= f; S[t][2] *= f; S[t][3] *= f; }
    }
    have_state = true;
#pragma unroll
    for (int kb = 0; kb < 4; ++kb) {
      uint32_t a[4], hi[4], lo[4];                   // value columns as rows: transposed fragments of V, decayed
      ldsm4_t(a, sV + (kb * 16 + (mi >> 1) * 8 + r8) * kLdV + warp * 16 + (mi & 1) * 8);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int j = kb * 16 + (q >> 1) * 8 + col2, d = m - 1 - j;            // rows beyond m hold zeros
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a[q]));
        split2(f.x * pw[d > 0 ? d : 0], f.y * pw[d > 1 ? d - 1 : 0], hi[q], lo[q]);
      }
#pragma unroll
      for (int t = 0; t < KB; t += 2) {
        uint32_t b[4], c[4];
        ldsm4_t(b, sK + (kb * 16 + (mi & 1) * 8 + r8) * LDK + t * 16 + (mi >> 1) * 8);
        ldsm4_t(c, sK + (kb * 16 + (mi & 1) * 8 + r8) * LDK + t * 16 + 16 + (mi >> 1) * 8);
        mma(S[2 * t], hi, b[0], b[1]);
        mma(S[2 * t + 1], hi, b[2], b[3]);
        mma(S[2 * t + 2], hi, c[0], c[1]);
        mma(S[2 * t + 3], hi, c[2], c[3]);
        mma(S[2 * t], lo, b[0], b[1]);
        mma(S[2 * t + 1], lo, b[2], b[3]);
        mma(S[2 * t + 2], lo, c[0], c[1]);
        mma(S[2 * t + 3], lo, c[2], c[3]);
      }
    }
  }
  if (slot >= 0) {
#pragma unroll
    for (int t = 0; t < 2 * KB; ++t)
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (vr + 8 * e < V)
          *reinterpret_cast<float2*>(st + static_cast<size_t>(vr + 8 * e) * DK + 8 * t + col2) = make_float2(S[t][2 * e], S[t][2 * e + 1]);
  }
}

template <int DK>
static int launch_chunk(const MbLightning& p, cudaStream_t stream) {
  constexpr int smem = (2 * kChunk * (2 * (DK + 8) + kLdV) + 2 * kChunk * kLdP) * 2;
  static PerDeviceOnce configured;
  if (configured.needed()) {
    if (cudaFuncSetAttribute(lightning_chunk_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return MB_ERR_LAUNCH;
    configured.done();
  }
  const int col_blocks = (p.vdim + kNV - 1) / kNV;
  return launch_plain(lightning_chunk_kernel<DK>, dim3(p.heads * col_blocks, p.B), dim3(kThreads), static_cast<size_t>(smem), stream, p,
                      col_blocks) == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

// sigmoid of an output gate: fp32 runs take the accurate exponential, 16-bit runs (the result is rounded) the fast one
template <typename T>
__device__ __forceinline__ float gate_of(float z) {
  if constexpr (sizeof(T) == 4) return sigmoidf(z);
  return __fdividef(1.f, 1.f + __expf(-z));
}

// o[t, :] = o / rms(o over the `n` true columns) * w * sigmoid(gate), in place; padding columns hold zeros
template <typename T>
__global__ void __launch_bounds__(1024) lightning_norm_kernel(T* __restrict__ o, int ldo, const T* __restrict__ gate, int ldg,
                                                              const T* __restrict__ w, int cols, int n, float eps) {
  constexpr int kHeld = 4;                           // 4-wide pieces a thread keeps in registers; more are read again
  __shared__ float part[32];
  const size_t t = blockIdx.x;
  T* row = o + t * ldo;
  const T* g = gate + t * ldg;
  float4 v[kHeld], b[kHeld];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kHeld; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    v[i] = c < cols ? ld4(row + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    b[i] = c < cols ? ld4(g + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
  }
  for (int c = (threadIdx.x + kHeld * blockDim.x) * 4; c < cols; c += blockDim.x * 4) {
    const float4 e = ld4(row + c);
    ss += e.x * e.x + e.y * e.y + e.z * e.z + e.w * e.w;
  }
  ss = warp_allsum(ss);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < static_cast<int>(blockDim.x >> 5); ++i) tot += part[i];
  const float inv = 1.f / sqrtf(tot / static_cast<float>(n) + eps);
  auto put = [&](int c, float4 e, float4 gt) {
    const float4 a = ld4(w + c);
    st4(row + c, make_float4(e.x * inv * a.x * gate_of<T>(gt.x), e.y * inv * a.y * gate_of<T>(gt.y), e.z * inv * a.z * gate_of<T>(gt.z),
                             e.w * inv * a.w * gate_of<T>(gt.w)));
  };
#pragma unroll
  for (int i = 0; i < kHeld; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    if (c < cols) put(c, v[i], b[i]);
  }
  for (int c = (threadIdx.x + kHeld * blockDim.x) * 4; c < cols; c += blockDim.x * 4) put(c, ld4(row + c), ld4(g + c));
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
  // 16-byte loads of every head's row; steps of one token per sequence are bound by the state and stay on the scan
  if (dtype == kBf16 && !p->one_token && p->dim_pad <= 128 && p->dim % 8 == 0 && p->vdim % 8 == 0 && p->ldx % 8 == 0 && p->q_off % 8 == 0 &&
      p->k_off % 8 == 0 && p->v_off % 8 == 0 && p->ldo % 2 == 0 && (reinterpret_cast<uintptr_t>(p->x) & 15) == 0 &&
      (reinterpret_cast<uintptr_t>(p->o) & 3) == 0) {
    switch (p->dim_pad) {
      case 32: return lightning::launch_chunk<32>(*p, stream);
      case 64: return lightning::launch_chunk<64>(*p, stream);
      case 96: return lightning::launch_chunk<96>(*p, stream);
      default: return lightning::launch_chunk<128>(*p, stream);
    }
  }
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
