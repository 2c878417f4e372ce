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

extern "C" int mb_gla(const MbGla* p, int dtype, int num_sms, cudaStream_t stream) {
  if (p->T <= 0 || p->B <= 0) return MB_OK;
  if (p->heads <= 0 || p->dim <= 0 || p->vdim <= 0 || p->dim % 8 || p->vdim % 8 || p->dim_pad != mb_delta_dim_pad(p->dim) || p->B > 65535 ||
      p->ldx % 8 || p->ldz % 4 || p->q_off % 8 || p->k_off % 8 || p->v_off % 8 || p->norm_dim <= 0 || p->norm_dim > p->vdim)
    return MB_ERR_SHAPE;
  if ((reinterpret_cast<uintptr_t>(p->x) | reinterpret_cast<uintptr_t>(p->z) | reinterpret_cast<uintptr_t>(p->z_bias) |
       reinterpret_cast<uintptr_t>(p->state) | reinterpret_cast<uintptr_t>(p->o)) & 15)
    return MB_ERR_ALIGN;
  return dtype == kF32 ? gla::run<float>(*p, num_sms, stream) : gla::run<__nv_bfloat16>(*p, num_sms, stream);
}
