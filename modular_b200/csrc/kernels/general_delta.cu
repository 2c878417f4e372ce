// Generalized delta rule (a decay and a removal rate per key channel and token) for ragged batches. Per head, with a state
// S [dim, vdim] in fp32, a key k and its unit vector u:
//   S <- (diag(w) - (a * u) u^T) S + k v^T;   o = S^T r;   w = exp(-exp(-1/2) sigmoid(z + w0)),  a = sigmoid(y + b)
// (both terms read the old state), and o is RMS-normed per head, scaled by a weight and gated.
//
//   general_delta_prep_kernel   one warp per (token, head): unit keys, decays and removal rates, all that enters the recurrence
//                               besides the values, in fp32: rows [u | w | -(a * u) | r], |k| and r . -(a * u)
//   general_delta_scan_kernel   columns of S are independent, so a warp owns 8 or 16 of them: eight lanes share the rows of a
//                               column (RL4 float4 each, in registers), four lane groups hold two or four columns each. With
//                               p = u . s and s' = w * s + u (|k| v), the new column is s' - (a * u) p and the output is
//                               r . s' - (r . (a * u)) p: both products are reduced together over the eight lanes, and one
//                               multiply-add per element waits for the reduction. Token rows are staged by cp.async, two chunks
//                               in flight. The state is read and written once per launch. In decode steps (one token per
//                               sequence) a CTA owns a whole head: its first warp makes the operands while the others load the
//                               state, and the output norm and gate are applied at the end. Longer steps leave fp32 outputs for
//                               mb_head_norm_gate.
//
// State: [slot, head, column, row], rows padded to a size the scan is built for; `state_idx[s]` is the sequence's slot
// (-1: start from zero and keep nothing), read when the step continues a sequence (kv_len > q_len).
#include <cuda_runtime.h>

#include "../common/api.h"
#include "../common/launch.h"
#include "../common/scalar.cuh"

namespace mb {
namespace gdelta {

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
__device__ __forceinline__ float dot4(float4 a, float4 b) { return a.x * b.x + a.y * b.y + a.z * b.z + a.w * b.w; }

constexpr float kDecayScale = -0.60653065971263342f;       // -exp(-1/2)

// Operands of one token and head, by one warp: [u | w | -(a * u) | r], every vector DP wide, then {|k|, r . -(a * u), 0, 0}.
template <typename T>
__device__ __forceinline__ void make_row(const MbGeneralDelta& p, size_t t, int h, float* __restrict__ dst) {
  const int lane = threadIdx.x & 31, D = p.dim, DP = p.dim_pad;
  const T* row = static_cast<const T*>(p.x) + t * p.ldx + h * D;
  float kk = 0.f, ra = 0.f;
  for (int c = lane * 4; c < D; c += 128) { const float4 k = ld4(row + p.k_off + c); kk += dot4(k, k); }
  const float len = sqrtf(warp_allsum(kk) + 1e-6f), inv = 1.f / len;
  for (int c = lane * 4; c < DP; c += 128) {
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f), w = u, au = u, r = u;
    if (c < D) {
      const float4 k = ld4(row + p.k_off + c), y = ld4(row + p.a_off + c), yb = *reinterpret_cast<const float4*>(p.a_bias + h * D + c);
      const float4 z = *reinterpret_cast<const float4*>(p.z + t * p.ldz + h * D + c),
                   zb = *reinterpret_cast<const float4*>(p.z_bias + h * D + c);
      r = ld4(row + p.r_off + c);
      u = make_float4(k.x * inv, k.y * inv, k.z * inv, k.w * inv);
      w = make_float4(expf(kDecayScale * sigmoidf(z.x + zb.x)), expf(kDecayScale * sigmoidf(z.y + zb.y)),
                      expf(kDecayScale * sigmoidf(z.z + zb.z)), expf(kDecayScale * sigmoidf(z.w + zb.w)));
      au = make_float4(-u.x * sigmoidf(y.x + yb.x), -u.y * sigmoidf(y.y + yb.y), -u.z * sigmoidf(y.z + yb.z), -u.w * sigmoidf(y.w + yb.w));
      ra += dot4(r, au);
    }
    *reinterpret_cast<float4*>(dst + c) = u;
    *reinterpret_cast<float4*>(dst + DP + c) = w;
    *reinterpret_cast<float4*>(dst + 2 * DP + c) = au;
    *reinterpret_cast<float4*>(dst + 3 * DP + c) = r;
  }
  ra = warp_allsum(ra);
  if (lane == 0) *reinterpret_cast<float4*>(dst + 4 * DP) = make_float4(len, ra, 0.f, 0.f);
}

template <typename T>
__global__ void __launch_bounds__(256) general_delta_prep_kernel(const MbGeneralDelta p) {
  const long long unit = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (unit >= static_cast<long long>(p.T) * p.heads) return;
  make_row<T>(p, static_cast<size_t>(unit / p.heads), static_cast<int>(unit % p.heads), p.rows + unit * (4 * p.dim_pad + 4));
}

template <typename T, int RL4, int NC, int MAXT, bool FUSE>
__global__ void __launch_bounds__(MAXT) general_delta_scan_kernel(const MbGeneralDelta p, int col_blocks, int chunk) {
  constexpr int DP = 32 * RL4, RF = 4 * DP + 4, E = 16 / static_cast<int>(sizeof(T));       // floats of a token row, values per copy
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float red[32];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = lane & 7, cg = lane >> 3, nt = blockDim.x;
  const int H = p.heads, V = p.vdim, cols = (nt >> 5) * 4 * NC;
  const int h = blockIdx.x / col_blocks, cbase = (blockIdx.x % col_blocks) * cols, s = blockIdx.y;
  const int t0 = p.q_start[s], n = p.q_len[s], slot = p.state_idx[s];
  if (n <= 0) return;
  const bool resume = slot >= 0 && p.kv_len[s] > n;
  const T* x = static_cast<const T*>(p.x);
  const size_t stage = static_cast<size_t>(chunk) * (RF * sizeof(float) + cols * sizeof(T));
  float* so = reinterpret_cast<float*>(smem + (FUSE ? 1 : 2) * stage);      // FUSE: outputs of one token
  auto fetch = [&](int c0, uint8_t* dst) {
    const int m = min(chunk, n - c0), vv = cols / E;
    float* rows = reinterpret_cast<float*>(dst);
    T* vals = reinterpret_cast<T*>(dst + static_cast<size_t>(chunk) * RF * sizeof(float));
    if (!FUSE) {
      const float* src = p.rows + (static_cast<size_t>(t0 + c0) * H + h) * RF;
      for (int i = tid; i < RF / 4; i += nt)
        for (int j = 0; j < m; ++j) cp_async16(rows + j * RF + i * 4, src + static_cast<size_t>(j) * H * RF + i * 4);
    }
    for (int i = tid; i < m * vv; i += nt) {
      const int j = i / vv, c = (i % vv) * E;
      if (cbase + c < V) cp_async16(vals + j * cols + c, x + static_cast<size_t>(t0 + c0 + j) * p.ldx + p.v_off + h * V + cbase + c);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, smem);
  const int lc = (warp * 4 + cg) * NC, col0 = cbase + lc;
  float* st = p.state + ((static_cast<size_t>(slot >= 0 ? slot : 0) * H + h) * V + col0) * DP;
  u64x2 S[NC][RL4];
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int i = 0; i < RL4; ++i)
      S[c][i] = (resume && col0 + c < V) ? *reinterpret_cast<const u64x2*>(st + c * DP + (i * 8 + rg) * 4) : u64x2{0ull, 0ull};
  if (FUSE && warp == 0) make_row<T>(p, t0, h, reinterpret_cast<float*>(smem));
  // which reduced value this lane ends up with: column `mine` of its group, key product or output
  const bool b4 = (lane & 4) != 0, b2 = (lane & 2) != 0, b1 = (lane & 1) != 0;
  const int mine = NC == 4 ? (b4 ? 2 : 0) + (b2 ? 1 : 0) : (b4 ? 1 : 0);
  const bool holds_o = NC == 4 ? b1 : (lane & 3) == 2;
  const bool writes = holds_o && col0 + mine < V;
  float* optr = FUSE ? nullptr : p.o + (static_cast<size_t>(t0) * H + h) * V + col0 + mine;
  for (int c0 = 0, it = 0; c0 < n; c0 += chunk, ++it) {
    const int m = min(chunk, n - c0);
    const uint8_t* buf = smem + (it & 1) * stage;
    if (c0 + chunk < n) {
      fetch(c0 + chunk, smem + ((it + 1) & 1) * stage);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float* rows = reinterpret_cast<const float*>(buf);
    const T* vals = reinterpret_cast<const T*>(buf + static_cast<size_t>(chunk) * RF * sizeof(float));
#pragma unroll 2
    for (int j = 0; j < m; ++j) {
      const float* rp = rows + j * RF;
      const float len = rp[4 * DP], ra = rp[4 * DP + 1];
      u64x2 au[RL4];
      uint64_t a[NC][2], b[NC][2], kv[NC];
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        a[c][0] = a[c][1] = b[c][0] = b[c][1] = 0ull;
        const float f = col0 + c < V ? len * ldf(vals + j * cols + lc + c) : 0.f;
        kv[c] = pack2(f, f);
      }
#pragma unroll
      for (int i = 0; i < RL4; ++i) {
        const int r = (i * 8 + rg) * 4;
        const u64x2 u4 = *reinterpret_cast<const u64x2*>(rp + r), w4 = *reinterpret_cast<const u64x2*>(rp + DP + r),
                    r4 = *reinterpret_cast<const u64x2*>(rp + 3 * DP + r);
        au[i] = *reinterpret_cast<const u64x2*>(rp + 2 * DP + r);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          a[c][0] = fma2(S[c][i].x, u4.x, a[c][0]); a[c][1] = fma2(S[c][i].y, u4.y, a[c][1]);
          S[c][i].x = fma2(S[c][i].x, w4.x, mul2(u4.x, kv[c])); S[c][i].y = fma2(S[c][i].y, w4.y, mul2(u4.y, kv[c]));
          b[c][0] = fma2(S[c][i].x, r4.x, b[c][0]); b[c][1] = fma2(S[c][i].y, r4.y, b[c][1]);
        }
      }
      float A[NC], B[NC];
#pragma unroll
      for (int c = 0; c < NC; ++c) { A[c] = sum4(a[c][0], a[c][1]); B[c] = sum4(b[c][0], b[c][1]); }
      // partial sums over the eight row lanes: every exchange halves the values a lane still carries
      float red8;
      if (NC == 4) {
        float a2[2], q2[2];
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          a2[c] = (b4 ? A[NC / 2 + c] : A[c]) + __shfl_xor_sync(0xffffffffu, b4 ? A[c] : A[NC / 2 + c], 4);
          q2[c] = (b4 ? B[NC / 2 + c] : B[c]) + __shfl_xor_sync(0xffffffffu, b4 ? B[c] : B[NC / 2 + c], 4);
        }
        const float a1 = (b2 ? a2[1] : a2[0]) + __shfl_xor_sync(0xffffffffu, b2 ? a2[0] : a2[1], 2);
        const float q1 = (b2 ? q2[1] : q2[0]) + __shfl_xor_sync(0xffffffffu, b2 ? q2[0] : q2[1], 2);
        red8 = (b1 ? q1 : a1) + __shfl_xor_sync(0xffffffffu, b1 ? a1 : q1, 1);
      } else {
        const float a1 = (b4 ? A[1] : A[0]) + __shfl_xor_sync(0xffffffffu, b4 ? A[0] : A[1], 4);
        const float q1 = (b4 ? B[1] : B[0]) + __shfl_xor_sync(0xffffffffu, b4 ? B[0] : B[1], 4);
        red8 = (b2 ? q1 : a1) + __shfl_xor_sync(0xffffffffu, b2 ? a1 : q1, 2);
        red8 += __shfl_xor_sync(0xffffffffu, red8, 1);
      }
      float pc[NC], p_mine = 0.f;                // u . s of this group's columns, from the lanes that hold them
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        pc[c] = __shfl_sync(0xffffffffu, red8, (lane & 24) | (NC == 4 ? (c >> 1) * 4 + (c & 1) * 2 : c * 4));
        p_mine = mine == c ? pc[c] : p_mine;
      }
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const uint64_t pp = pack2(pc[c], pc[c]);
#pragma unroll
        for (int i = 0; i < RL4; ++i) { S[c][i].x = fma2(au[i].x, pp, S[c][i].x); S[c][i].y = fma2(au[i].y, pp, S[c][i].y); }
      }
      const float o = fmaf(p_mine, ra, red8);    // in the lanes that hold an output
      if (!FUSE) {
        if (writes) *optr = o;
        optr += H * V;
      } else {                                   // one CTA holds the whole head (cbase = 0)
        if (holds_o) so[lc + mine] = col0 + mine < V ? o : 0.f;
        __syncthreads();
        float ss = 0.f;
        for (int c = tid; c < V; c += nt) ss = fmaf(so[c], so[c], ss);
        ss = warp_allsum(ss);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        float tot = 0.f;
        for (int i = 0; i < (nt >> 5); ++i) tot += red[i];
        const float inv = 1.f / sqrtf(tot / static_cast<float>(p.norm_dim) + p.eps);
        const size_t t = static_cast<size_t>(t0);
        for (int c = tid; c < V; c += nt) {
          const float g = ldf(static_cast<const T*>(p.gate) + t * p.ld_gate + h * V + c);
          stf(static_cast<T*>(p.out) + t * p.ld_out + h * V + c, so[c] * inv * ldf(static_cast<const T*>(p.norm_w) + h * V + c) * sigmoidf(g));
        }
      }
    }
    if (!FUSE) __syncthreads();                  // the stage is free again
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
static int scan_launch(const MbGeneralDelta& p, int warps, bool fuse, cudaStream_t stream) {
  constexpr int MAXT = RL4 <= 8 ? 512 : 256;
  const int cols = warps * 4 * NC, col_blocks = (p.vdim + cols - 1) / cols;
  const int per_token = (4 * 32 * RL4 + 4) * 4 + cols * static_cast<int>(sizeof(T));
  int chunk = fuse ? 1 : 44 * 1024 / (2 * per_token);
  chunk = chunk > 16 ? 16 : chunk < 1 ? 1 : chunk;
  const size_t smem = static_cast<size_t>(fuse ? 1 : 2) * chunk * per_token + (fuse ? cols * 4 : 0);
  if (smem > 48 * 1024 - 256) return MB_ERR_TOO_LARGE;
  const dim3 grid(p.heads * col_blocks, p.B), block(warps * 32);
  const cudaError_t e = fuse ? launch_plain(general_delta_scan_kernel<T, RL4, NC, MAXT, true>, grid, block, smem, stream, p, col_blocks, chunk)
                             : launch_plain(general_delta_scan_kernel<T, RL4, NC, MAXT, false>, grid, block, smem, stream, p, col_blocks, chunk);
  return e == cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
}

template <typename T, int RL4>
static int scan(const MbGeneralDelta& p, int num_sms, cudaStream_t stream) {
  constexpr int max_warps = (RL4 <= 8 ? 512 : 256) / 32;
  const int head_warps = (p.vdim + 7) / 8;
  if (p.one_token && head_warps <= max_warps) return scan_launch<T, RL4, 2>(p, head_warps, true, stream);
  if (launch_plain(general_delta_prep_kernel<T>, dim3(static_cast<unsigned>((static_cast<long long>(p.T) * p.heads + 7) / 8)), dim3(256), 0,
                   stream, p) != cudaSuccess)
    return MB_ERR_LAUNCH;
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
  if (rc != MB_OK) return rc;
  const MbHeadOut o = {p.o, p.out, p.ld_out, p.gate, p.ld_gate, p.norm_w, p.T, p.heads, p.vdim, p.norm_dim, 0, p.eps, 1.f, p.vdim};
  return mb_head_norm_gate(&o, sizeof(T) == 4 ? kF32 : kBf16, stream);
}

template <typename T>
static int run(const MbGeneralDelta& p, int num_sms, cudaStream_t stream) {
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

}  // namespace gdelta
}  // namespace mb

using namespace mb;

extern "C" int mb_general_delta(const MbGeneralDelta* p, int dtype, int num_sms, cudaStream_t stream) {
  if (p->T <= 0 || p->B <= 0) return MB_OK;
  if (p->heads <= 0 || p->dim <= 0 || p->dim % 8 || p->vdim <= 0 || p->vdim % 8 || p->dim_pad != mb_delta_dim_pad(p->dim) || p->ldx % 8 ||
      p->r_off % 8 || p->k_off % 8 || p->v_off % 8 || p->a_off % 8 || p->ldz % 4 || p->norm_dim <= 0 || p->norm_dim > p->vdim)
    return MB_ERR_SHAPE;
  if ((reinterpret_cast<uintptr_t>(p->x) | reinterpret_cast<uintptr_t>(p->z) | reinterpret_cast<uintptr_t>(p->z_bias) |
       reinterpret_cast<uintptr_t>(p->a_bias) | reinterpret_cast<uintptr_t>(p->rows) | reinterpret_cast<uintptr_t>(p->state)) & 15)
    return MB_ERR_ALIGN;
  return dtype == kF32 ? gdelta::run<float>(*p, num_sms, stream) : gdelta::run<__nv_bfloat16>(*p, num_sms, stream);
}
