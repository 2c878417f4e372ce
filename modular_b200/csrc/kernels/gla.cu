// Gated linear attention (a decay per key channel and token) for ragged batches. Per head, with a state S [dim, vdim] in fp32:
//   S <- diag(alpha) S + k v^T;   o = S^T q;   alpha = sigmoid(z + bias)^(1 / tau)
// and the output is RMS-normed per head, scaled by a weight and gated.
//
//   gla_scan_kernel   token by token on the CUDA cores, everything in fp32. Columns of S are independent, so a warp owns
//                     4 NC of them: eight lanes share the rows of a column (RL4 float4 each, in registers). Raw rows of the
//                     next chunk of tokens travel by cp.async while this one is worked on; a pass over shared memory turns
//                     them into fp32 operands (the decay's logarithm and exponential included) once per chunk. The state is
//                     read and written once per launch. Decode steps give a CTA a whole head, which then also applies the
//                     norm and the gate; longer sequences leave fp32 outputs for mb_head_norm_gate.
//   gla_intra_kernel  bf16 prompts, 64 tokens at a time on the tensor cores; everything that does not need the state, for all
//                     chunks at once. With b the running sum of log alpha inside a chunk and its four blocks of 16 tokens,
//                       o_i  = sum_{j <= i} (q_i exp(b_i - b_j)) . k_j  v_j        (this kernel)
//                            + S^T (q_i exp(b_i))                                  (the next one, S: state before the chunk)
//                       S'   = diag(exp(b_last)) S + sum_j (k_j exp(b_last - b_j)) v_j^T
//                     Only decays relative to a block's edge are formed, q_i exp(b_i - r_I) and k_j exp(r_J+1 - b_j) with r_I the
//                     sum ahead of block I, both at most 1; products of blocks multiply them by exp(r_I - r_J+1) <= 1. Inside a
//                     block the factor is exp(r_I - r_I+1), at least 1: where it would pass exp(64) for some channel, the block's
//                     products are made from running products of alpha instead. All of this is fp32 and enters a product as the
//                     sum of two bf16 numbers (three products of halves, relative error about 2^-16).
//   gla_state_kernel  walks the chunks of one (sequence, head, 64 value columns) with S^T in the accumulator fragments of the
//                     warp that owns its 16 columns, which are also the B fragments of S^T q; adds its part to the outputs.
//
// State: [slot, head, column, row], rows padded to a size the scan is built for; `state_idx[s]` is the sequence's slot
// (-1: start from zero and keep nothing), read when the step continues a sequence (kv_len > q_len).
#include <cuda_runtime.h>

#include "../common/api.h"
#include "../common/launch.h"
#include "../common/scalar.cuh"

namespace mb {
namespace gla {

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src)
               : "memory");
}

// two fp32 lanes per 64-bit register
struct __align__(16) u64x2 { uint64_t x, y; };
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float sum4(uint64_t a, uint64_t b) {
  float x, y;
  uint64_t c;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(c) : "l"(a), "l"(b));
  asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(c));
  return x + y;
}

// logarithm of the decay: log sigmoid(y) / tau
__device__ __forceinline__ float log_decay(float y, float inv_tau) { return (fminf(y, 0.f) - log1pf(expf(-fabsf(y)))) * inv_tau; }

// The same for the chunk kernels, whose operands keep 16 to 17 bits: relative error of a few 1e-7 plus 1e-7 per unit of |y|
__device__ __forceinline__ float log_decay_fast(float y, float inv_tau) { return (fminf(y, 0.f) - log1pf(__expf(-fabsf(y)))) * inv_tau; }

template <typename T, int RL4, int NC, int MAXT, bool FUSE>
__global__ void __launch_bounds__(MAXT) gla_scan_kernel(const MbGla p, int col_blocks, int chunk) {
  constexpr int DP = 32 * RL4, E = 16 / static_cast<int>(sizeof(T));       // elements per 16-byte copy
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float red[32];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = lane & 7, cg = lane >> 3, nt = blockDim.x;
  const int H = p.heads, V = p.vdim, D = p.dim, cols = (nt >> 5) * 4 * NC;
  const int h = blockIdx.x / col_blocks, cbase = (blockIdx.x % col_blocks) * cols, s = blockIdx.y;
  const int t0 = p.q_start[s], n = p.q_len[s], slot = p.state_idx[s];
  if (n <= 0) return;
  const bool resume = slot >= 0 && p.kv_len[s] > n;
  const int row_floats = 3 * DP + cols;                    // q | k | alpha | v columns of a token, fp32
  float* work = reinterpret_cast<float*>(smem);
  const int raw_z = chunk * D, raw_x = chunk * (2 * D + cols);              // raw stage: z fp32 [chunk][D]; q | k [D], v [cols]
  const size_t raw_bytes = raw_z * sizeof(float) + raw_x * sizeof(T);
  uint8_t* raw = smem + static_cast<size_t>(chunk) * row_floats * sizeof(float);
  float* so = reinterpret_cast<float*>(raw + 2 * raw_bytes);                // FUSE: outputs of one token
  const T* x = static_cast<const T*>(p.x);
  const int vcols = min(cols, V - cbase);
  auto fetch = [&](int c0, uint8_t* dst) {
    const int m = min(chunk, n - c0), qv = D / E, vv = vcols / E, per = 2 * qv + vv;
    float* dz = reinterpret_cast<float*>(dst);
    T* dx = reinterpret_cast<T*>(dst + raw_z * sizeof(float));
    for (int i = tid; i < m * (D / 4); i += nt) {
      const int j = i / (D / 4), c = (i % (D / 4)) * 4;
      cp_async16(dz + j * D + c, p.z + static_cast<size_t>(t0 + c0 + j) * p.ldz + h * D + c);
    }
    for (int i = tid; i < m * per; i += nt) {
      const int j = i / per, k = i % per;
      const T* row = x + static_cast<size_t>(t0 + c0 + j) * p.ldx;
      T* d = dx + j * (2 * D + cols);
      if (k < qv) cp_async16(d + k * E, row + p.q_off + h * D + k * E);
      else if (k < 2 * qv) cp_async16(d + k * E, row + p.k_off + h * D + (k - qv) * E);
      else cp_async16(d + 2 * D + (k - 2 * qv) * E, row + p.v_off + h * V + cbase + (k - 2 * qv) * E);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, raw);
  const int lc = (warp * 4 + cg) * NC, col0 = cbase + lc;
  float* st = p.state + ((static_cast<size_t>(slot >= 0 ? slot : 0) * H + h) * V + col0) * DP;
  u64x2 S[NC][RL4];
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int i = 0; i < RL4; ++i)
      S[c][i] = (resume && col0 + c < V) ? *reinterpret_cast<const u64x2*>(st + c * DP + (i * 8 + rg) * 4) : u64x2{0ull, 0ull};
  const bool b4 = (lane & 4) != 0, b2 = (lane & 2) != 0;
  const int mine = NC == 4 ? (b4 ? 2 : 0) + (b2 ? 1 : 0) : (b4 ? 1 : 0);    // the column whose sum this lane ends up with
  const bool holds = NC == 4 ? (lane & 1) == 0 : (lane & 3) == 0;
  const bool writes = holds && col0 + mine < V;
  for (int c0 = 0, it = 0; c0 < n; c0 += chunk, ++it) {
    const int m = min(chunk, n - c0);
    const uint8_t* src = raw + (it & 1) * raw_bytes;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                       // this chunk is in; the last one's operands are done with
    if (c0 + chunk < n) fetch(c0 + chunk, raw + ((it + 1) & 1) * raw_bytes);
    {
      const float* sz = reinterpret_cast<const float*>(src);
      const T* sx = reinterpret_cast<const T*>(src + raw_z * sizeof(float));
      const int per = row_floats / 4;
      for (int i = tid; i < m * per; i += nt) {
        const int j = i / per, c = (i % per) * 4;
        const T* xr = sx + j * (2 * D + cols);
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < DP) {
          if (c < D) { v = ld4(xr + c); v.x *= p.q_scale; v.y *= p.q_scale; v.z *= p.q_scale; v.w *= p.q_scale; }
        } else if (c < 2 * DP) {
          if (c - DP < D) v = ld4(xr + D + c - DP);
        } else if (c < 3 * DP) {
          const int ch = c - 2 * DP;
          if (ch < D) {
            const float4 a = *reinterpret_cast<const float4*>(sz + j * D + ch);
            const float4 b = *reinterpret_cast<const float4*>(p.z_bias + h * D + ch);
            v = make_float4(expf(log_decay(a.x + b.x, p.inv_tau)), expf(log_decay(a.y + b.y, p.inv_tau)),
                            expf(log_decay(a.z + b.z, p.inv_tau)), expf(log_decay(a.w + b.w, p.inv_tau)));
          }
        } else if (c - 3 * DP < vcols) {
          v = ld4(xr + 2 * D + c - 3 * DP);
        }
        *reinterpret_cast<float4*>(work + j * row_floats + c) = v;
      }
    }
    __syncthreads();
#pragma unroll 2
    for (int j = 0; j < m; ++j) {
      const float* rp = work + j * row_floats;
      uint64_t a[NC][2], vv[NC];
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        a[c][0] = a[c][1] = 0ull;
        const float f = rp[3 * DP + lc + c];
        vv[c] = pack2(f, f);
      }
#pragma unroll
      for (int i = 0; i < RL4; ++i) {
        const int r = (i * 8 + rg) * 4;
        const u64x2 q4 = *reinterpret_cast<const u64x2*>(rp + r), k4 = *reinterpret_cast<const u64x2*>(rp + DP + r),
                    g4 = *reinterpret_cast<const u64x2*>(rp + 2 * DP + r);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          S[c][i].x = fma2(S[c][i].x, g4.x, mul2(k4.x, vv[c])); S[c][i].y = fma2(S[c][i].y, g4.y, mul2(k4.y, vv[c]));
          a[c][0] = fma2(S[c][i].x, q4.x, a[c][0]); a[c][1] = fma2(S[c][i].y, q4.y, a[c][1]);
        }
      }
      float A[NC];
#pragma unroll
      for (int c = 0; c < NC; ++c) A[c] = sum4(a[c][0], a[c][1]);
      // partial sums over the eight row lanes: every exchange halves the values a lane still carries
      float o;
      if (NC == 4) {
        float a2[2];
#pragma unroll
        for (int c = 0; c < 2; ++c) a2[c] = (b4 ? A[NC / 2 + c] : A[c]) + __shfl_xor_sync(0xffffffffu, b4 ? A[c] : A[NC / 2 + c], 4);
        o = (b2 ? a2[1] : a2[0]) + __shfl_xor_sync(0xffffffffu, b2 ? a2[0] : a2[1], 2);
        o += __shfl_xor_sync(0xffffffffu, o, 1);
      } else {
        o = (b4 ? A[1] : A[0]) + __shfl_xor_sync(0xffffffffu, b4 ? A[0] : A[1], 4);
        o += __shfl_xor_sync(0xffffffffu, o, 2);
        o += __shfl_xor_sync(0xffffffffu, o, 1);
      }
      const size_t t = static_cast<size_t>(t0 + c0 + j);
      if (!FUSE) {
        if (writes) p.o[(t * H + h) * V + col0 + mine] = o;
      } else {                                             // one CTA holds the whole head (cbase = 0)
        if (holds) so[lc + mine] = col0 + mine < V ? o : 0.f;
        __syncthreads();
        float ss = 0.f;
        for (int c = tid; c < V; c += nt) ss = fmaf(so[c], so[c], ss);
        ss = warp_allsum(ss);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        float tot = 0.f;
        for (int i = 0; i < (nt >> 5); ++i) tot += red[i];
        const float inv = p.out_mult / sqrtf(tot / static_cast<float>(p.norm_dim) + p.eps);
        for (int c = tid; c < V; c += nt) {
          const float g = ldf(static_cast<const T*>(p.gate) + t * p.ld_gate + h * V + c);
          stf(static_cast<T*>(p.out) + t * p.ld_out + h * V + c,
              so[c] * inv * ldf(static_cast<const T*>(p.norm_w) + c) * (p.gate_silu ? siluf(g) : sigmoidf(g)));
        }
        __syncthreads();
      }
    }
  }
  if (slot >= 0) {
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int i = 0; i < RL4; ++i)
        if (col0 + c < V) *reinterpret_cast<u64x2*>(st + c * DP + (i * 8 + rg) * 4) = S[c][i];
  }
}

template <typename T, int RL4, int NC>
static int scan_launch(const MbGla& p, int warps, bool fuse, cudaStream_t stream) {
  constexpr int MAXT = RL4 <= 8 ? 512 : 256;
  const int cols = warps * 4 * NC, col_blocks = (p.vdim + cols - 1) / cols;
  const int work = (3 * 32 * RL4 + cols) * 4, raw = p.dim * 4 + (2 * p.dim + cols) * static_cast<int>(sizeof(T));
  int chunk = p.one_token ? 1 : 44 * 1024 / (work + 2 * raw);
  chunk = chunk > 16 ? 16 : chunk < 1 ? 1 : chunk;
  const size_t smem = static_cast<size_t>(chunk) * (work + 2 * raw) + (fuse ? cols * 4 : 0);
  if (smem > 48 * 1024 - 256) return MB_ERR_TOO_LARGE;
  const dim3 grid(p.heads * col_blocks, p.B), block(warps * 32);
  const cudaError_t e = fuse ? launch_plain(gla_scan_kernel<T, RL4, NC, MAXT, true>, grid, block, smem, stream, p, col_blocks, chunk)
                             : launch_plain(gla_scan_kernel<T, RL4, NC, MAXT, false>, grid, block, smem, stream, p, col_blocks, chunk);
  return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

static int finish(const MbGla& p, int dtype, cudaStream_t stream) {
  const MbHeadOut o = {p.o, p.out, p.ld_out, p.gate, p.ld_gate, p.norm_w, p.T, p.heads, p.vdim, p.norm_dim, p.gate_silu, p.eps, p.out_mult};
  return mb_head_norm_gate(&o, dtype, stream);
}

template <typename T, int RL4>
static int scan(const MbGla& p, int num_sms, cudaStream_t stream) {
  constexpr int max_warps = (RL4 <= 8 ? 512 : 256) / 32;
  const int head_warps = (p.vdim + 7) / 8;
  if (p.one_token && head_warps <= max_warps) return scan_launch<T, RL4, 2>(p, head_warps, true, stream);
  // longer sequences: four columns per lane where the registers allow it, and CTAs of up to four warps as long as the grid has
  // one per SM
  auto fit = [&](int per_warp) {
    const int hw = (p.vdim + per_warp - 1) / per_warp;
    int w = hw < 4 ? hw : 4;
    while (w > 1 && static_cast<long long>(p.B) * p.heads * ((hw + w - 1) / w) < num_sms) w >>= 1;
    return w;
  };
  int rc = MB_ERR_SHAPE;
  if constexpr (RL4 <= 4) {
    if (p.vdim >= 16) rc = scan_launch<T, RL4, 4>(p, fit(16), false, stream);
    else rc = scan_launch<T, RL4, 2>(p, fit(8), false, stream);
  } else {
    rc = scan_launch<T, RL4, 2>(p, fit(8), false, stream);
  }
  return rc != MB_OK ? rc : finish(p, sizeof(T) == 4 ? kF32 : kBf16, stream);
}

// ---------------------------------------------------------------------------- chunks on the tensor cores
typedef __nv_bfloat16 bf16;
constexpr int kC = 64, kSub = 16, kThreads = 128;      // tokens per chunk and block; four warps, one block of rows each
constexpr float kWide = 64.f;                          // largest decay inside a block, as an exponent, that factors are made for

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void cp_async16z(void* dst, const void* src, bool valid) {
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
__device__ __forceinline__ float2 unpack2(uint32_t v) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v)); }

template <int DK>
struct IntraSmem {
  static constexpr int LDQ = DK + 4, LDK = DK + 8;
  float q[kC * LDQ];                  // q_i exp(b_i - r_I)
  bf16 kh[kC * LDK], kl[kC * LDK];    // k_j exp(r_J+1 - b_j)
  float tot[4][DK];                   // sum of log alpha over a block
  float diag[4][DK];                  // exp(r_I - r_I+1)
  float far[3][DK];                   // exp(r_I - r_J+1) for (I, J) = (2, 0), (3, 0), (3, 1)
  float head[3][DK], tail[3][DK];     // exp(r_I), I = 1 .. 3;  exp(b_last - r_J+1), J = 0 .. 2
  float exact[4][kSub][kSub + 1];     // products inside a block with a wide decay
  int wide[4];                        // a block has one
};

// Products of block I with the blocks at or before it, then times the values.
template <int I, int DK>
__device__ __forceinline__ void intra_rows(const MbGla& p, IntraSmem<DK>& sm, const bf16* sV, int ldv, size_t t0, int h, int m, int wide) {
  constexpr int LDQ = IntraSmem<DK>::LDQ, LDK = IntraSmem<DK>::LDK;
  const int lane = threadIdx.x & 31, mi = lane >> 3, r8 = lane & 7, row4 = lane >> 2, col2 = 2 * (lane & 3);
  float acc[I + 1][2][4];
#pragma unroll
  for (int J = 0; J <= I; ++J)
#pragma unroll
    for (int n = 0; n < 2; ++n) acc[J][n][0] = acc[J][n][1] = acc[J][n][2] = acc[J][n][3] = 0.f;
#pragma unroll 2
  for (int kb = 0; kb < DK / 16; ++kb) {
    const int c = kb * 16 + col2;
    const float *r0 = sm.q + (I * kSub + row4) * LDQ + c, *r1 = r0 + 8 * LDQ;
    const float2 x[4] = {*reinterpret_cast<const float2*>(r0), *reinterpret_cast<const float2*>(r1),
                         *reinterpret_cast<const float2*>(r0 + 8), *reinterpret_cast<const float2*>(r1 + 8)};
#pragma unroll
    for (int J = 0; J <= I; ++J) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      if (J == I - 1) {
#pragma unroll
        for (int i = 0; i < 4; ++i) split2(x[i].x, x[i].y, ah[i], al[i]);
      } else {
        const float* f = J == I ? sm.diag[I] : I == 2 ? sm.far[0] : J == 0 ? sm.far[1] : sm.far[2];
        const float2 f0 = *reinterpret_cast<const float2*>(f + c), f1 = *reinterpret_cast<const float2*>(f + c + 8);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 g = i < 2 ? f0 : f1;
          split2(x[i].x * g.x, x[i].y * g.y, ah[i], al[i]);
        }
      }
      const int off = (J * kSub + (mi >> 1) * 8 + r8) * LDK + kb * 16 + (mi & 1) * 8;
      ldsm4(bh, sm.kh + off);
      ldsm4(bl, sm.kl + off);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        mma(acc[J][n], ah, bh[2 * n], bh[2 * n + 1]);
        mma(acc[J][n], al, bh[2 * n], bh[2 * n + 1]);
        mma(acc[J][n], ah, bl[2 * n], bl[2 * n + 1]);
      }
    }
  }
#pragma unroll
  for (int n = 0; n < 2; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = row4 + 8 * (e >> 1), j = n * 8 + col2 + (e & 1);
      if (j > i) acc[I][n][e] = 0.f;
      else if (wide) acc[I][n][e] = sm.exact[I][i][j];
    }
  uint32_t ph[I + 1][4], pl[I + 1][4];
#pragma unroll
  for (int J = 0; J <= I; ++J)
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      split2(acc[J][n][0], acc[J][n][1], ph[J][2 * n], pl[J][2 * n]);
      split2(acc[J][n][2], acc[J][n][3], ph[J][2 * n + 1], pl[J][2 * n + 1]);
    }
  const int V = p.vdim, HV = p.heads * V;
  float* out = p.o + (t0 + I * kSub + row4) * HV + h * V;
  const bool on0 = I * kSub + row4 < m, on1 = I * kSub + row4 + 8 < m;
  for (int v0 = 0; v0 < V; v0 += 16) {
    float o[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int J = 0; J <= I; ++J) {
      uint32_t b[4];
      ldsm4_t(b, sV + (J * kSub + (mi & 1) * 8 + r8) * ldv + v0 + (mi >> 1) * 8);
#pragma unroll
      for (int n = 0; n < 2; ++n) { mma(o[n], ph[J], b[2 * n], b[2 * n + 1]); mma(o[n], pl[J], b[2 * n], b[2 * n + 1]); }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const int c = v0 + n * 8 + col2;
      if (c >= V) continue;
      if (on0) *reinterpret_cast<float2*>(out + c) = make_float2(o[n][0], o[n][1]);
      if (on1) *reinterpret_cast<float2*>(out + 8 * HV + c) = make_float2(o[n][2], o[n][3]);
    }
  }
}

template <int DK>
__global__ void __launch_bounds__(kThreads, 2) gla_intra_kernel(const MbGla p) {
  constexpr int LDQ = IntraSmem<DK>::LDQ, LDK = IntraSmem<DK>::LDK;
  extern __shared__ __align__(16) uint8_t smem[];
  IntraSmem<DK>& sm = *reinterpret_cast<IntraSmem<DK>*>(smem);
  bf16* sV = reinterpret_cast<bf16*>(smem + sizeof(IntraSmem<DK>));
  static_assert(sizeof(IntraSmem<DK>) % 16 == 0, "the values follow");
  const int tile = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int s = p.tile_seq[tile];
  if (s < 0) return;
  if (tid < 4) sm.wide[tid] = 0;
  const int c0 = p.tile_q0[tile], m = min(kC, p.q_len[s] - c0), D = p.dim, V = p.vdim, V16 = (V + 15) & ~15, ldv = V16 + 8;
  const size_t t0 = static_cast<size_t>(p.q_start[s]) + c0;
  const bf16* x = static_cast<const bf16*>(p.x) + t0 * p.ldx;
  for (int i = tid; i < kC * (V16 / 8); i += kThreads) {        // rows beyond the sequence and columns beyond the head: zeros
    const int j = i / (V16 / 8), c = (i % (V16 / 8)) * 8;
    const bool ok = j < m && c < V;
    cp_async16z(sV + j * ldv + c, ok ? x + static_cast<size_t>(j) * p.ldx + p.v_off + h * V + c : x, ok);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  for (int u = tid; u < 4 * (DK / 2); u += kThreads) {          // one block of 16 tokens and two channels
    const int I = u / (DK / 2), c = (u % (DK / 2)) * 2;
    const bool on = c < D;
    const float* z = p.z + (t0 + I * kSub) * p.ldz + h * D + c;
    const bf16* row = x + static_cast<size_t>(I * kSub) * p.ldx + h * D + c;
    float2 bias = make_float2(0.f, 0.f);
    if (on) bias = *reinterpret_cast<const float2*>(p.z_bias + h * D + c);
    float2 b[kSub], run = make_float2(0.f, 0.f);
    uint32_t q[kSub], k[kSub];
#pragma unroll
    for (int i = 0; i < kSub; ++i) {
      b[i] = make_float2(0.f, 0.f);
      q[i] = k[i] = 0u;
      if (!on || I * kSub + i >= m) continue;
      b[i] = *reinterpret_cast<const float2*>(z + static_cast<size_t>(i) * p.ldz);
      q[i] = *reinterpret_cast<const uint32_t*>(row + static_cast<size_t>(i) * p.ldx + p.q_off);
      k[i] = *reinterpret_cast<const uint32_t*>(row + static_cast<size_t>(i) * p.ldx + p.k_off);
    }
#pragma unroll
    for (int i = 0; i < kSub; ++i) {
      if (on && I * kSub + i < m) {
        run.x += log_decay_fast(b[i].x + bias.x, p.inv_tau);
        run.y += log_decay_fast(b[i].y + bias.y, p.inv_tau);
      }
      b[i] = run;
    }
    *reinterpret_cast<float2*>(&sm.tot[I][c]) = run;
#pragma unroll
    for (int i = 0; i < kSub; ++i) {
      const float2 qv = unpack2(q[i]), kv = unpack2(k[i]);
      const int r = I * kSub + i;
      *reinterpret_cast<float2*>(sm.q + r * LDQ + c) = make_float2(qv.x * p.q_scale * __expf(b[i].x), qv.y * p.q_scale * __expf(b[i].y));
      uint32_t hi, lo;
      split2(kv.x * __expf(run.x - b[i].x), kv.y * __expf(run.y - b[i].y), hi, lo);
      *reinterpret_cast<uint32_t*>(sm.kh + r * LDK + c) = hi;
      *reinterpret_cast<uint32_t*>(sm.kl + r * LDK + c) = lo;
    }
  }
  __syncthreads();
  const size_t unit = static_cast<size_t>(tile) * p.heads + h;
  if (tid < DK) {
    const int c = tid;
    const float a0 = sm.tot[0][c], a1 = sm.tot[1][c], a2 = sm.tot[2][c], a3 = sm.tot[3][c];
#pragma unroll
    for (int I = 0; I < 4; ++I) {
      const float a = sm.tot[I][c];
      const bool w = -a > kWide;
      if (w) sm.wide[I] = 1;
      sm.diag[I][c] = w ? 0.f : expf(-a);
    }
    sm.far[0][c] = expf(a1); sm.far[1][c] = expf(a1 + a2); sm.far[2][c] = expf(a2);
    sm.head[0][c] = expf(a0); sm.head[1][c] = expf(a0 + a1); sm.head[2][c] = expf(a0 + a1 + a2);
    sm.tail[0][c] = expf(a1 + a2 + a3); sm.tail[1][c] = expf(a2 + a3); sm.tail[2][c] = expf(a3);
    p.ends[unit * DK + c] = expf(a0 + a1 + a2 + a3);
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  // what the state kernel multiplies: q_i exp(b_i) and k_j exp(b_last - b_j), halves apart
  bf16* qk = static_cast<bf16*>(p.qk) + unit * 4 * kC * DK;
  for (int i = tid; i < kC * (DK / 4); i += kThreads) {
    const int r = i / (DK / 4), c = (i % (DK / 4)) * 4, I = r / kSub;
    float4 q = *reinterpret_cast<const float4*>(sm.q + r * LDQ + c);
    if (I > 0) {
      const float4 f = *reinterpret_cast<const float4*>(&sm.head[I - 1][c]);
      q.x *= f.x; q.y *= f.y; q.z *= f.z; q.w *= f.w;
    }
    uint2 hi = *reinterpret_cast<const uint2*>(sm.kh + r * LDK + c), lo = *reinterpret_cast<const uint2*>(sm.kl + r * LDK + c);
    if (I < 3) {
      const float4 f = *reinterpret_cast<const float4*>(&sm.tail[I][c]);
      const float2 a = unpack2(hi.x), al = unpack2(lo.x), b = unpack2(hi.y), bl = unpack2(lo.y);
      split2((a.x + al.x) * f.x, (a.y + al.y) * f.y, hi.x, lo.x);
      split2((b.x + bl.x) * f.z, (b.y + bl.y) * f.w, hi.y, lo.y);
    }
    uint2 qh, ql;
    split2(q.x, q.y, qh.x, ql.x);
    split2(q.z, q.w, qh.y, ql.y);
    const size_t o = static_cast<size_t>(r) * DK + c;
    *reinterpret_cast<uint2*>(qk + o) = qh;
    *reinterpret_cast<uint2*>(qk + kC * DK + o) = ql;
    *reinterpret_cast<uint2*>(qk + 2 * kC * DK + o) = hi;
    *reinterpret_cast<uint2*>(qk + 3 * kC * DK + o) = lo;
  }
  const bool mine_wide = sm.wide[warp] != 0;
  if (mine_wide) {                                   // this warp's block: running products, lanes share the channels
    constexpr int CL = DK / 32;
    float al[kSub][CL];
#pragma unroll
    for (int i = 0; i < kSub; ++i)
#pragma unroll
      for (int e = 0; e < CL; ++e) {
        const int c = lane + 32 * e, r = warp * kSub + i;
        al[i][e] = c < D && r < m ? expf(log_decay(p.z[(t0 + r) * p.ldz + h * D + c] + p.z_bias[h * D + c], p.inv_tau)) : 1.f;
      }
    for (int j = 0; j < kSub; ++j) {
      const int rj = warp * kSub + j;
      float w[CL];
#pragma unroll
      for (int e = 0; e < CL; ++e) {
        const int c = lane + 32 * e;
        w[e] = c < D && rj < m ? ldf(x + static_cast<size_t>(rj) * p.ldx + p.k_off + h * D + c) : 0.f;
      }
#pragma unroll
      for (int i = 0; i < kSub; ++i) {
        if (i < j) continue;
        const int ri = warp * kSub + i;
        float a = 0.f;
#pragma unroll
        for (int e = 0; e < CL; ++e) {
          const int c = lane + 32 * e;
          if (i > j) w[e] *= al[i][e];
          if (c < D && ri < m) a = fmaf(ldf(x + static_cast<size_t>(ri) * p.ldx + p.q_off + h * D + c) * p.q_scale, w[e], a);
        }
        a = warp_allsum(a);
        if (lane == 0) sm.exact[warp][i][j] = a;
      }
    }
    __syncwarp();
  }
  switch (warp) {
    case 0: intra_rows<0, DK>(p, sm, sV, ldv, t0, h, m, mine_wide); break;
    case 1: intra_rows<1, DK>(p, sm, sV, ldv, t0, h, m, mine_wide); break;
    case 2: intra_rows<2, DK>(p, sm, sV, ldv, t0, h, m, mine_wide); break;
    default: intra_rows<3, DK>(p, sm, sV, ldv, t0, h, m, mine_wide); break;
  }
}

constexpr int kNV = 64, kLdV = kNV + 8;

template <int DK>
struct StateStage {
  static constexpr int LDK = DK + 8;
  bf16 qk[4][kC * LDK];               // q hi, q lo, k hi, k lo
  bf16 v[kC * kLdV];
  float end[DK];
};

// One CTA walks the chunks of one (sequence, head, 64 value columns).
template <int DK>
__global__ void __launch_bounds__(kThreads, 1) gla_state_kernel(const MbGla p, int col_blocks) {
  constexpr int LDK = StateStage<DK>::LDK, KB = DK / 16;
  extern __shared__ __align__(16) uint8_t smem[];
  StateStage<DK>* stages = reinterpret_cast<StateStage<DK>*>(smem);
  __shared__ int first_tile;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mi = lane >> 3, r8 = lane & 7, row4 = lane >> 2, col2 = 2 * (lane & 3);
  const int h = blockIdx.x / col_blocks, v0 = (blockIdx.x % col_blocks) * kNV, s = blockIdx.y, H = p.heads, V = p.vdim;
  const int n = p.q_len[s], slot = p.state_idx[s];
  if (n <= 0) return;
  if (warp == 0) {                                   // chunks lie sequence by sequence
    int f = 0;
    for (int b = lane; b < s; b += 32) f += (p.q_len[b] + kC - 1) / kC;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) f += __shfl_xor_sync(0xffffffffu, f, o);
    if (lane == 0) first_tile = f;
  }
  __syncthreads();
  const size_t t0 = p.q_start[s], tile0 = first_tile;
  const bool resume = slot >= 0 && p.kv_len[s] > n;
  const bf16* x = static_cast<const bf16*>(p.x) + t0 * p.ldx + p.v_off + h * V + v0;
  auto fetch = [&](int it, StateStage<DK>& st) {
    const size_t unit = (tile0 + it) * H + h;
    const bf16* src = static_cast<const bf16*>(p.qk) + unit * 4 * kC * DK;
    constexpr int CH = DK / 8;
    for (int i = tid; i < 4 * kC * CH; i += kThreads) {
      const int a = i / (kC * CH), j = i / CH % kC, c = (i % CH) * 8;
      cp_async16(&st.qk[a][j * LDK + c], src + (static_cast<size_t>(a) * kC + j) * DK + c);
    }
    for (int i = tid; i < kC * (kNV / 8); i += kThreads) {
      const int j = i / (kNV / 8), c = (i % (kNV / 8)) * 8;
      const bool ok = it * kC + j < n && v0 + c < V;
      cp_async16z(st.v + j * kLdV + c, ok ? x + static_cast<size_t>(it * kC + j) * p.ldx + c : x, ok);
    }
    if (tid < DK / 4) cp_async16(st.end + tid * 4, p.ends + unit * DK + tid * 4);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, stages[0]);
  // S^T: 16 value columns of this warp as accumulator tiles of 8 keys: [0], [1] value row4, [2], [3] value row4 + 8
  float S[2 * KB][4];
  float* st = p.state + (static_cast<size_t>(slot >= 0 ? slot : 0) * H + h) * V * DK;
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
  for (int c0 = 0, it = 0; c0 < n; c0 += kC, ++it) {
    const int m = min(kC, n - c0);
    const StateStage<DK>& sg = stages[it & 1];
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                 // this chunk is in, the last one is done with its stage
    if (c0 + kC < n) fetch(it + 1, stages[(it + 1) & 1]);
    if (have_state) {                                // S^T q for all queries and this warp's 16 value columns
      float o[4][2][4];
      float2 was[4][2][2];                           // what the other kernel left; read while the products run
      float* out = p.o + (t0 + c0 + row4) * H * V + h * V + v0 + warp * 16 + col2;
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;
#pragma unroll
          for (int e = 0; e < 2; ++e)
            if (i * 16 + row4 + 8 * e < m && v0 + warp * 16 + j * 8 + col2 < V)
              was[i][j][e] = *reinterpret_cast<const float2*>(out + static_cast<size_t>(i * 16 + 8 * e) * H * V + j * 8);
        }
#pragma unroll
      for (int kb = 0; kb < KB; ++kb) {
        uint32_t hi[2][2], lo[2][2];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e) split2(S[2 * kb + e][2 * j], S[2 * kb + e][2 * j + 1], hi[j][e], lo[j][e]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          uint32_t a[4], b[4];
          const int off = (i * 16 + (lane & 15)) * LDK + kb * 16 + (lane >> 4) * 8;
          ldsm4(a, sg.qk[0] + off);
          ldsm4(b, sg.qk[1] + off);
          mma(o[i][0], a, hi[0][0], hi[0][1]); mma(o[i][1], a, hi[1][0], hi[1][1]);
          mma(o[i][0], b, hi[0][0], hi[0][1]); mma(o[i][1], b, hi[1][0], hi[1][1]);
          mma(o[i][0], a, lo[0][0], lo[0][1]); mma(o[i][1], a, lo[1][0], lo[1][1]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e)
            if (i * 16 + row4 + 8 * e < m && v0 + warp * 16 + j * 8 + col2 < V)
              *reinterpret_cast<float2*>(out + static_cast<size_t>(i * 16 + 8 * e) * H * V + j * 8) =
                  make_float2(was[i][j][e].x + o[i][j][2 * e], was[i][j][e].y + o[i][j][2 * e + 1]);
#pragma unroll
      for (int t = 0; t < 2 * KB; ++t) {
        const float2 f = *reinterpret_cast<const float2*>(sg.end + 8 * t + col2);
        S[t][0] *= f.x; S[t][1] *= f.y; S[t][2] *= f.x; S[t][3] *= f.y;
      }
    }
    have_state = true;
#pragma unroll
    for (int kb = 0; kb < 4; ++kb) {
      uint32_t a[4];                                 // value columns as rows: transposed fragments of V
      ldsm4_t(a, sg.v + (kb * 16 + (mi >> 1) * 8 + r8) * kLdV + warp * 16 + (mi & 1) * 8);
#pragma unroll
      for (int t = 0; t < KB; ++t) {
        uint32_t b[4], c[4];
        const int off = (kb * 16 + (mi & 1) * 8 + r8) * LDK + t * 16 + (mi >> 1) * 8;
        ldsm4_t(b, sg.qk[2] + off);
        ldsm4_t(c, sg.qk[3] + off);
        mma(S[2 * t], a, b[0], b[1]);
        mma(S[2 * t + 1], a, b[2], b[3]);
        mma(S[2 * t], a, c[0], c[1]);
        mma(S[2 * t + 1], a, c[2], c[3]);
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
static int launch_chunks(const MbGla& p, cudaStream_t stream) {
  const size_t intra = sizeof(IntraSmem<DK>) + static_cast<size_t>(kC) * (((p.vdim + 15) & ~15) + 8) * sizeof(bf16);
  const size_t state = 2 * sizeof(StateStage<DK>);
  static PerDeviceOnce configured;
  if (configured.needed()) {
    if (cudaFuncSetAttribute(gla_intra_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024) != cudaSuccess ||
        cudaFuncSetAttribute(gla_state_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(state)) != cudaSuccess)
      return MB_ERR_LAUNCH;
    configured.done();
  }
  if (intra > 160 * 1024) return MB_ERR_TOO_LARGE;
  if (launch_plain(gla_intra_kernel<DK>, dim3(p.n_tiles, p.heads), dim3(kThreads), intra, stream, p) != cudaSuccess) return MB_ERR_LAUNCH;
  const int col_blocks = (p.vdim + kNV - 1) / kNV;
  if (launch_plain(gla_state_kernel<DK>, dim3(p.heads * col_blocks, p.B), dim3(kThreads), state, stream, p, col_blocks) != cudaSuccess)
    return MB_ERR_LAUNCH;
  return finish(p, kBf16, stream);
}

template <typename T>
static int run(const MbGla& p, int num_sms, cudaStream_t stream) {
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

}  // namespace gla
}  // namespace mb

using namespace mb;

// Chunks of a step at most, or 0 where it runs token by token: fp32, wide heads, steps of a few tokens per sequence.
extern "C" int mb_gla_chunks(const MbGla* p, int dtype) {
  if (dtype != kBf16 || p->one_token || p->dim_pad > 128 || p->vdim > 256 || p->heads > 65535 || p->T < 64 || p->T < 8 * p->B) return 0;
  return p->T / gla::kC + p->B;
}

extern "C" int mb_gla(const MbGla* p, int dtype, int num_sms, cudaStream_t stream) {
  if (p->T <= 0 || p->B <= 0) return MB_OK;
  if (p->heads <= 0 || p->dim <= 0 || p->vdim <= 0 || p->dim % 8 || p->vdim % 8 || p->dim_pad != mb_delta_dim_pad(p->dim) || p->B > 65535 ||
      p->ldx % 8 || p->ldz % 4 || p->q_off % 8 || p->k_off % 8 || p->v_off % 8 || p->norm_dim <= 0 || p->norm_dim > p->vdim)
    return MB_ERR_SHAPE;
  if ((reinterpret_cast<uintptr_t>(p->x) | reinterpret_cast<uintptr_t>(p->z) | reinterpret_cast<uintptr_t>(p->z_bias) |
       reinterpret_cast<uintptr_t>(p->state) | reinterpret_cast<uintptr_t>(p->o)) & 15)
    return MB_ERR_ALIGN;
  if (p->n_tiles > 0 && p->qk != nullptr) {
    if (dtype != kBf16 || p->dim_pad > 128 || p->vdim > 256) return MB_ERR_SHAPE;
    if ((reinterpret_cast<uintptr_t>(p->qk) | reinterpret_cast<uintptr_t>(p->ends)) & 15) return MB_ERR_ALIGN;
    switch (p->dim_pad) {
      case 32: return gla::launch_chunks<32>(*p, stream);
      case 64: return gla::launch_chunks<64>(*p, stream);
      case 96: return gla::launch_chunks<96>(*p, stream);
      default: return gla::launch_chunks<128>(*p, stream);
    }
  }
  return dtype == kF32 ? gla::run<float>(*p, num_sms, stream) : gla::run<__nv_bfloat16>(*p, num_sms, stream);
}
