// Gated delta rule with a decay per key channel or per head, for ragged batches. Per head, with a state S [dim, vdim] in
// fp32:
//   S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
// q, k and v pass a short causal convolution and silu first, q and k are unit vectors per head, and o is RMS-normed over
// vdim, scaled by a weight and gated.
//
//   delta_prep_kernel   one warp per (token, piece): convolution + silu of q, k, v (inputs before the step come from the
//                       sequence's convolution state), unit norms, decays g = exp(-exp(A_log) softplus(z + dt_bias)),
//                       beta, k . q. Everything leaves in fp32.
//   delta_scan_kernel   columns of S are independent, so a warp owns 8 or 16 of them: eight lanes share the rows of a
//                       column (each 4 * RL4 of them, in registers), four lane groups hold two or four columns each. A
//                       token costs one pass of decay, two dot products per column reduced together over eight lanes
//                       (o = (gS)^T q + u (k . q) needs no second reduction), and the rank-one update. Token rows are
//                       staged through shared memory with cp.async. The state is read once and written once per launch,
//                       [slot, head, column, row]; sequences of one token are a decode step, for which one CTA owns a
//                       whole head and also applies the output norm and gate. The convolution state is advanced at the
//                       end of this kernel, after every read of it by the first one.
//   head_out_kernel     output norm and gate for longer sequences, one warp per (token, head)
//
// A chunked formulation on the tensor cores would round what enters the recurrence to 16 bits; this one keeps it in fp32.
#include <cuda_runtime.h>

#include "../common/api.h"
#include "../common/launch.h"
#include "../common/scalar.cuh"

namespace mb {
namespace delta {

__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src)
               : "memory");
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src)
               : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// two fp32 lanes per 64-bit register: one instruction for two multiply-adds, each rounded like fmaf
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

// silu of a convolution output: fp32 runs take the accurate exponential, 16-bit runs the fast one
template <typename T>
__device__ __forceinline__ float conv_act(float z) {
  if constexpr (sizeof(T) == 4) return siluf(z);
  return __fdividef(z, 1.f + __expf(-z));
}

__device__ __forceinline__ float softplusf(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// factor of the output gate: fp32 runs take the accurate exponential, 16-bit runs (the result is rounded) the fast one
template <typename T>
__device__ __forceinline__ float gate_of(float z, int silu, float mult) {
  if constexpr (sizeof(T) == 4) return mult * (silu ? siluf(z) : sigmoidf(z));
  return __fdividef(silu ? mult * z : mult, 1.f + __expf(-z));
}

// units of the preparation that make decays and step sizes: one per head, or 32 heads together with one decay per head
__device__ __host__ __forceinline__ int decay_units(const MbDelta& p) { return p.z ? p.heads : (p.heads + 31) / 32; }
template <typename T>
__device__ __forceinline__ void head_decay(const MbDelta& p, const T* row, int t, int h) {
  if (h >= p.heads) return;
  const size_t i = static_cast<size_t>(t) * p.heads + h;
  p.g[i] = expf(-expf(p.A_log[h]) * softplusf(ldf(row + p.a_off + h) + p.dt_bias[h]));
  p.beta[i] = sigmoidf(ldf(row + p.b_off + h));
}

template <typename T>
__global__ void __launch_bounds__(256) delta_prep_kernel(const MbDelta p) {
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  const int unit = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int KH = p.kv_heads, H = p.heads, D = p.dim, V = p.vdim, DP = p.dim_pad;
  const int qkC = KH * D, vC = H * V, C = 2 * qkC + vC, W = p.taps;
  const int v_units = (vC + 127) / 128, G = decay_units(p);
  if (unit >= KH + G + v_units) return;
  int s = t;
  if (!p.one_token) {
    int lo = 0, hi = p.B - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (p.q_start[mid] <= t) lo = mid; else hi = mid - 1;
    }
    s = lo;
  }
  const int off = t - p.q_start[s];
  if (off < 0 || off >= p.q_len[s]) return;      // a row of no sequence
  const T* row = static_cast<const T*>(p.x) + static_cast<size_t>(t) * p.ldx;
  const int slot = p.state_idx[s];
  const float* hist = (slot >= 0 && W > 1 && p.kv_len[s] > p.q_len[s])
                          ? p.conv_state + static_cast<size_t>(slot) * C * (W - 1) : nullptr;
  // channel `ch` of the convolution state, read from column `col` of the projection rows
  auto conv_silu = [&](int ch, int col) {
    const T* w = static_cast<const T*>(p.conv_w) + static_cast<size_t>(ch) * W;
    float acc = 0.f;
    for (int j = 0; j < W; ++j) {
      const int src = off - (W - 1) + j;
      float xv = 0.f;
      if (src >= 0) xv = ldf(row - static_cast<ptrdiff_t>(W - 1 - j) * p.ldx + col);
      else if (hist) xv = hist[static_cast<size_t>(ch) * (W - 1) + (W - 1 + src)];
      acc = fmaf(ldf(w + j), xv, acc);
    }
    return siluf(acc);
  };
  if (unit < KH) {
    float* qo = p.q + (static_cast<size_t>(t) * KH + unit) * DP;
    float* ko = p.k + (static_cast<size_t>(t) * KH + unit) * DP;
    float qq = 0.f, kk = 0.f, kq = 0.f;
    for (int c = lane; c < D; c += 32) {
      const float a = conv_silu(unit * D + c, p.q_off + unit * D + c);
      const float b = conv_silu(qkC + unit * D + c, p.k_off + unit * D + c);
      qq = fmaf(a, a, qq); kk = fmaf(b, b, kk); kq = fmaf(a, b, kq);
      qo[c] = a; ko[c] = b;                        // rescaled below by the same lane
    }
    qq = warp_allsum(qq); kk = warp_allsum(kk); kq = warp_allsum(kq);
    const float iq = 1.f / sqrtf(qq + 1e-6f) / sqrtf(static_cast<float>(D)), ik = 1.f / sqrtf(kk + 1e-6f);
    for (int c = lane; c < DP; c += 32) {
      qo[c] = c < D ? qo[c] * iq : 0.f;
      ko[c] = c < D ? ko[c] * ik : 0.f;
    }
    if (lane == 0) p.kq[static_cast<size_t>(t) * KH + unit] = kq * iq * ik;
  } else if (unit < KH + G && !p.z) {
    head_decay(p, row, t, (unit - KH) * 32 + lane);
  } else if (unit < KH + G) {
    const int h = unit - KH;
    const float a = expf(p.A_log[h]);
    const float* z = p.z + static_cast<size_t>(t) * p.ldz + h * D;
    float* go = p.g + (static_cast<size_t>(t) * H + h) * DP;
    for (int c = lane; c < DP; c += 32) go[c] = c < D ? expf(-a * softplusf(z[c] + p.dt_bias[h * D + c])) : 0.f;
    if (lane == 0) p.beta[static_cast<size_t>(t) * H + h] = sigmoidf(ldf(row + p.b_off + h));
  } else {
    const int c0 = (unit - KH - G) * 128;
    for (int c = c0 + lane; c < min(c0 + 128, vC); c += 32)
      p.v[static_cast<size_t>(t) * vC + c] = conv_silu(2 * qkC + c, p.v_off + c);
  }
}

// The same for key widths up to 128 (a multiple of 4) and W taps known at compile time: a lane owns four neighbouring
// channels, keeps its taps and the convolution window in registers and walks `tile` consecutive tokens.
template <int W>
struct ConvLane {
  float w[W][4];
  float4 win[W];                    // the last W - 1 inputs in win[1..]
  template <typename T>
  __device__ __forceinline__ void taps(const T* p) {     // [4 channels, W]
#pragma unroll
    for (int c = 0; c < 4; ++c)
#pragma unroll
      for (int j = 0; j < W; ++j) w[j][c] = ldf(p + c * W + j);
  }
  // inputs before token `off` of its sequence: rows of the step, then the state (`hist` [4 channels, W - 1] or none)
  template <typename T>
  __device__ __forceinline__ void start(const T* x, int ldx, int off, const float* hist) {
#pragma unroll
    for (int j = 0; j < W - 1; ++j) {
      const int src = off - (W - 1) + j;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (src >= 0) {
        v = ld4(x - static_cast<ptrdiff_t>(W - 1 - j) * ldx);
      } else if (hist) {
        const float* h = hist + (W - 1 + src);
        v = make_float4(h[0], h[W - 1], h[2 * (W - 1)], h[3 * (W - 1)]);
      }
      win[j + 1] = v;
    }
  }
  template <typename T>
  __device__ __forceinline__ float4 step(float4 x) {
#pragma unroll
    for (int j = 0; j < W - 1; ++j) win[j] = win[j + 1];
    win[W - 1] = x;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < W; ++j) {
      a.x = fmaf(w[j][0], win[j].x, a.x); a.y = fmaf(w[j][1], win[j].y, a.y);
      a.z = fmaf(w[j][2], win[j].z, a.z); a.w = fmaf(w[j][3], win[j].w, a.w);
    }
    return make_float4(conv_act<T>(a.x), conv_act<T>(a.y), conv_act<T>(a.z), conv_act<T>(a.w));
  }
};

template <typename T, int W>
__global__ void __launch_bounds__(256) delta_prep_fast_kernel(const MbDelta p, int tile) {
  const int lane = threadIdx.x & 31;
  const int unit = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int KH = p.kv_heads, H = p.heads, D = p.dim, V = p.vdim, DP = p.dim_pad;
  const int qkC = KH * D, vC = H * V, C = 2 * qkC + vC;
  const int G = decay_units(p);
  if (unit >= KH + G + (vC + 127) / 128) return;
  const int tb = blockIdx.x * tile, te = min(tb + tile, p.T);
  int s = tb;
  if (!p.one_token) {
    int lo = 0, hi = p.B - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (p.q_start[mid] <= tb) lo = mid; else hi = mid - 1;
    }
    s = lo;
  }
  const bool is_qk = unit < KH, is_g = !is_qk && unit < KH + G;
  const int c = lane * 4;
  const int v0 = is_qk || is_g ? 0 : (unit - KH - G) * 128;
  const bool on = is_qk || is_g ? c < D : v0 + c < vC;
  const T* w = static_cast<const T*>(p.conv_w);
  const T* xq = static_cast<const T*>(p.x) + (is_qk ? p.q_off + unit * D + c : p.v_off + v0 + c);
  const T* xk = static_cast<const T*>(p.x) + p.k_off + unit * D + c;
  const int ch_a = is_qk ? unit * D + c : 2 * qkC + v0 + c, ch_b = qkC + unit * D + c;
  ConvLane<W> ca, cb;
  if (on && !is_g) ca.taps(w + static_cast<size_t>(ch_a) * W);
  if (on && is_qk) cb.taps(w + static_cast<size_t>(ch_b) * W);
  const bool chan_g = is_g && p.z;
  const float a_log = chan_g ? expf(p.A_log[unit - KH]) : 0.f;
  float4 bias = make_float4(0.f, 0.f, 0.f, 0.f);
  if (chan_g && on) bias = *reinterpret_cast<const float4*>(p.dt_bias + (unit - KH) * D + c);
  const float scale = 1.f / sqrtf(static_cast<float>(D));
  float4 fut_a = make_float4(0.f, 0.f, 0.f, 0.f), fut_b = fut_a;
  if (on && !is_g) fut_a = ld4(xq + static_cast<size_t>(tb) * p.ldx);
  if (on && is_qk) fut_b = ld4(xk + static_cast<size_t>(tb) * p.ldx);
  int end = 0;                       // first token behind the current sequence
  for (int t = tb; t < te; ++t) {
    if (t >= end) {                  // a new sequence (or the first token of the tile)
      if (t > tb) ++s;
      while (s < p.B && p.q_start[s] + p.q_len[s] <= t) ++s;
      if (s >= p.B || p.q_start[s] > t) return;      // rows of no sequence
      end = p.q_start[s] + p.q_len[s];
      if (!is_g && on) {
        const int off = t - p.q_start[s], slot = p.state_idx[s];
        const float* hist = (slot >= 0 && W > 1 && p.kv_len[s] > p.q_len[s])
                                ? p.conv_state + static_cast<size_t>(slot) * C * (W - 1) : nullptr;
        ca.start(xq + static_cast<size_t>(t) * p.ldx, p.ldx, off, hist ? hist + static_cast<size_t>(ch_a) * (W - 1) : nullptr);
        if (is_qk)
          cb.start(xk + static_cast<size_t>(t) * p.ldx, p.ldx, off, hist ? hist + static_cast<size_t>(ch_b) * (W - 1) : nullptr);
      }
    }
    const size_t row = static_cast<size_t>(t) * p.ldx;
    const float4 nxt_a = fut_a, nxt_b = fut_b;
    if (on && t + 1 < te) {          // the next token's inputs travel while this one is worked on
      if (!is_g) fut_a = ld4(xq + row + p.ldx);
      if (is_qk) fut_b = ld4(xk + row + p.ldx);
    }
    if (is_qk) {
      float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q;
      if (on) { q = ca.template step<T>(nxt_a); k = cb.template step<T>(nxt_b); }
      float qq = q.x * q.x + q.y * q.y + q.z * q.z + q.w * q.w, kk = k.x * k.x + k.y * k.y + k.z * k.z + k.w * k.w;
      float kq = q.x * k.x + q.y * k.y + q.z * k.z + q.w * k.w;
      qq = warp_allsum(qq); kk = warp_allsum(kk); kq = warp_allsum(kq);
      const float iq = scale / sqrtf(qq + 1e-6f), ik = 1.f / sqrtf(kk + 1e-6f);
      const size_t o = (static_cast<size_t>(t) * KH + unit) * DP + c;
      if (c < DP) {
        *reinterpret_cast<float4*>(p.q + o) = make_float4(q.x * iq, q.y * iq, q.z * iq, q.w * iq);
        *reinterpret_cast<float4*>(p.k + o) = make_float4(k.x * ik, k.y * ik, k.z * ik, k.w * ik);
      }
      if (lane == 0) p.kq[static_cast<size_t>(t) * KH + unit] = kq * iq * ik;
    } else if (is_g && !chan_g) {
      head_decay(p, static_cast<const T*>(p.x) + row, t, (unit - KH) * 32 + lane);
    } else if (is_g) {
      const int h = unit - KH;
      float4 g = make_float4(0.f, 0.f, 0.f, 0.f);
      if (on) {
        const float4 z = *reinterpret_cast<const float4*>(p.z + static_cast<size_t>(t) * p.ldz + h * D + c);
        g = make_float4(expf(-a_log * softplusf(z.x + bias.x)), expf(-a_log * softplusf(z.y + bias.y)),
                        expf(-a_log * softplusf(z.z + bias.z)), expf(-a_log * softplusf(z.w + bias.w)));
      }
      if (c < DP) *reinterpret_cast<float4*>(p.g + (static_cast<size_t>(t) * H + h) * DP + c) = g;
      if (lane == 0) p.beta[static_cast<size_t>(t) * H + h] = sigmoidf(ldf(static_cast<const T*>(p.x) + row + p.b_off + h));
    } else if (on) {
      *reinterpret_cast<float4*>(p.v + static_cast<size_t>(t) * vC + v0 + c) = ca.template step<T>(nxt_a);
    }
  }
}

template <typename T, int RL4, int NC, int MAXT, bool FUSE, bool HEADG>
__global__ void __launch_bounds__(MAXT) delta_scan_kernel(const MbDelta p, int col_blocks, int chunk) {
  constexpr int DP = 32 * RL4, NP = HEADG ? 2 : 3, NS = HEADG ? 4 : 2;     // fp32 vectors and scalars per token
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rg = lane & 7, cg = lane >> 3;
  const int KH = p.kv_heads, H = p.heads, V = p.vdim;
  const int h = blockIdx.x / col_blocks, cols = (blockDim.x >> 5) * 4 * NC, cbase = (blockIdx.x % col_blocks) * cols;
  const int kh = h / (H / KH), s = blockIdx.y;
  const int t0 = p.q_start[s], n = p.q_len[s], slot = p.state_idx[s];
  const bool resume = slot >= 0 && p.kv_len[s] > n;
  if (n > 0) {
    const int row_floats = NP * DP + cols;         // q | k | (g) | v columns, then beta, k . q (and g) per token
    const int stage_floats = chunk * (row_floats + NS);
    float* so = sm + 2 * stage_floats;             // FUSE: outputs of one token
    auto fetch = [&](int c0, float* dst) {         // every thread walks the tokens of its piece of the row
      const int m = min(chunk, n - c0);
      const size_t t = static_cast<size_t>(t0 + c0);
      for (int pc = tid; pc < NP * DP / 4; pc += blockDim.x) {
        const int which = pc / (DP / 4), c = (pc % (DP / 4)) * 4;
        const float* src = which == 0 ? p.q + (t * KH + kh) * DP : which == 1 ? p.k + (t * KH + kh) * DP : p.g + (t * H + h) * DP;
        src += c;
        const int step = (which == 2 ? H : KH) * DP;
        float* d = dst + pc * 4;
        for (int j = 0; j < m; ++j, src += step, d += row_floats) cp_async16(d, src);
      }
      if (tid < cols && cbase + tid < V) {
        const float* src = p.v + (t * H + h) * V + cbase + tid;
        float* d = dst + NP * DP + tid;
        for (int j = 0; j < m; ++j, src += H * V, d += row_floats) cp_async4(d, src);
      }
      float* sc = dst + chunk * row_floats;
      for (int i = tid; i < NS * m; i += blockDim.x) {
        const int k = i % NS;
        if (k < 3) cp_async4(sc + i, k == 1 ? p.kq + (t + i / NS) * KH + kh : (k == 0 ? p.beta : p.g) + (t + i / NS) * H + h);
      }
      cp_async_commit();
    };
    fetch(0, sm);
    const int col0 = cbase + (warp * 4 + cg) * NC;
    float* st = p.state + ((static_cast<size_t>(slot >= 0 ? slot : 0) * H + h) * V + col0) * DP;
    u64x2 S[NC][RL4];                              // four rows per entry, two packed fp32 pairs
#pragma unroll
    for (int i = 0; i < RL4; ++i)
#pragma unroll
      for (int c = 0; c < NC; ++c)
        S[c][i] = (resume && col0 + c < V) ? *reinterpret_cast<const u64x2*>(st + c * DP + (i * 8 + rg) * 4) : u64x2{0ull, 0ull};
    // which reduced value this lane ends up with: column `mine` of its group, key product or query product
    const bool b4 = (lane & 4) != 0, b2 = (lane & 2) != 0, b1 = (lane & 1) != 0;
    const int mine = NC == 4 ? (b4 ? 2 : 0) + (b2 ? 1 : 0) : (b4 ? 1 : 0);
    const bool is_q = NC == 4 ? b1 : b2;
    const int my_col = (warp * 4 + cg) * NC + mine;
    float* optr = p.o + (static_cast<size_t>(t0) * H + h) * V + cbase + my_col;
    const bool holds_o = NC == 4 ? b1 : (lane & 3) == 2;
    const bool writes = holds_o && cbase + my_col < V;
    for (int c0 = 0, it = 0; c0 < n; c0 += chunk, ++it) {
      const int m = min(chunk, n - c0);
      const float* buf = sm + (it & 1) * stage_floats;
      if (c0 + chunk < n) { fetch(c0 + chunk, sm + ((it + 1) & 1) * stage_floats); cp_async_wait<1>(); } else { cp_async_wait<0>(); }
      __syncthreads();
      const float* sc = buf + chunk * row_floats;
#pragma unroll 2
      for (int j = 0; j < m; ++j) {
        const float* rowp = buf + j * row_floats;
        u64x2 kr[RL4];
        uint64_t a[NC][2], b[NC][2], gh = 0ull;
        if (HEADG) gh = pack2(sc[NS * j + 2], sc[NS * j + 2]);
#pragma unroll
        for (int c = 0; c < NC; ++c) a[c][0] = a[c][1] = b[c][0] = b[c][1] = 0ull;
#pragma unroll
        for (int i = 0; i < RL4; ++i) {
          const int r = (i * 8 + rg) * 4;
          const u64x2 q4 = *reinterpret_cast<const u64x2*>(rowp + r);
          const u64x2 k4 = *reinterpret_cast<const u64x2*>(rowp + DP + r);
          const u64x2 g4 = HEADG ? u64x2{gh, gh} : *reinterpret_cast<const u64x2*>(rowp + 2 * DP + r);
          kr[i] = k4;
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            S[c][i].x = mul2(S[c][i].x, g4.x); S[c][i].y = mul2(S[c][i].y, g4.y);
            a[c][0] = fma2(S[c][i].x, k4.x, a[c][0]); a[c][1] = fma2(S[c][i].y, k4.y, a[c][1]);
            b[c][0] = fma2(S[c][i].x, q4.x, b[c][0]); b[c][1] = fma2(S[c][i].y, q4.y, b[c][1]);
          }
        }
        float A[NC], Bq[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) { A[c] = sum4(a[c][0], a[c][1]); Bq[c] = sum4(b[c][0], b[c][1]); }
        // partial sums over the eight row lanes: every exchange halves the values a lane still carries
        float r;
        if (NC == 4) {
          float a2[2], q2[2];
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            a2[c] = (b4 ? A[NC / 2 + c] : A[c]) + __shfl_xor_sync(0xffffffffu, b4 ? A[c] : A[NC / 2 + c], 4);
            q2[c] = (b4 ? Bq[NC / 2 + c] : Bq[c]) + __shfl_xor_sync(0xffffffffu, b4 ? Bq[c] : Bq[NC / 2 + c], 4);
          }
          const float a1 = (b2 ? a2[1] : a2[0]) + __shfl_xor_sync(0xffffffffu, b2 ? a2[0] : a2[1], 2);
          const float q1 = (b2 ? q2[1] : q2[0]) + __shfl_xor_sync(0xffffffffu, b2 ? q2[0] : q2[1], 2);
          r = (b1 ? q1 : a1) + __shfl_xor_sync(0xffffffffu, b1 ? a1 : q1, 1);
        } else {
          const float a1 = (b4 ? A[1] : A[0]) + __shfl_xor_sync(0xffffffffu, b4 ? A[0] : A[1], 4);
          const float q1 = (b4 ? Bq[1] : Bq[0]) + __shfl_xor_sync(0xffffffffu, b4 ? Bq[0] : Bq[1], 4);
          r = (b2 ? q1 : a1) + __shfl_xor_sync(0xffffffffu, b2 ? a1 : q1, 2);
          r += __shfl_xor_sync(0xffffffffu, r, 1);
        }
        const float beta = sc[NS * j], kq = sc[NS * j + 1];
        const float vv = rowp[NP * DP + my_col];
        const float u = beta * (vv - r);           // meaningful in the lanes that hold a key product
        float uc[NC], u_mine = 0.f;
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          uc[c] = __shfl_sync(0xffffffffu, u, (lane & 24) | (NC == 4 ? (c >> 1) * 4 + (c & 1) * 2 : c * 4));
          u_mine = mine == c ? uc[c] : u_mine;
        }
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          const uint64_t up = pack2(uc[c], uc[c]);
#pragma unroll
          for (int i = 0; i < RL4; ++i) { S[c][i].x = fma2(kr[i].x, up, S[c][i].x); S[c][i].y = fma2(kr[i].y, up, S[c][i].y); }
        }
        const float o = fmaf(u_mine, kq, r);       // in the lanes that hold a query product
        if (FUSE) {
          if (holds_o) so[my_col] = cbase + my_col < V ? o : 0.f;
        } else {
          if (writes) *optr = o;
          optr += H * V;
        }
        if (FUSE) {                                // one CTA holds the whole head (cbase = 0)
          __syncthreads();
          float ss = 0.f;
          for (int c = tid; c < V; c += blockDim.x) ss = fmaf(so[c], so[c], ss);
          ss = warp_allsum(ss);
          if (lane == 0) red[warp] = ss;
          __syncthreads();
          float tot = 0.f;
          for (int i = 0; i < static_cast<int>(blockDim.x >> 5); ++i) tot += red[i];
          const float inv = 1.f / sqrtf(tot / static_cast<float>(V) + p.eps);
          const size_t t = static_cast<size_t>(t0 + c0 + j);
          for (int c = tid; c < V; c += blockDim.x) {
            const float gate = gate_of<T>(ldf(static_cast<const T*>(p.gate) + t * p.ld_gate + h * V + c), p.gate_silu, p.out_mult);
            stf(static_cast<T*>(p.out) + t * p.ld_out + h * V + c, so[c] * inv * ldf(static_cast<const T*>(p.norm_w) + c) * gate);
          }
          __syncthreads();
        }
      }
      __syncthreads();                             // the stage is free again
    }
    if (slot >= 0) {
#pragma unroll
      for (int i = 0; i < RL4; ++i)
#pragma unroll
        for (int c = 0; c < NC; ++c)
          if (col0 + c < V) *reinterpret_cast<u64x2*>(st + c * DP + (i * 8 + rg) * 4) = S[c][i];
    }
  }
  // the last taps - 1 convolution inputs of the sequence; this CTA's share of the channels
  const int W = p.taps;
  if (n > 0 && slot >= 0 && W > 1) {
    const int qkC = KH * p.dim, C = 2 * qkC + H * V;
    for (int c = blockIdx.x * blockDim.x + tid; c < C; c += gridDim.x * blockDim.x) {
      const int col = c < qkC ? p.q_off + c : c < 2 * qkC ? p.k_off + (c - qkC) : p.v_off + (c - 2 * qkC);
      float* cs = p.conv_state + (static_cast<size_t>(slot) * C + c) * (W - 1);
      // ascending order only overwrites entries that have been read: entry i comes from entry i + n
      for (int i = 0; i < W - 1; ++i) {
        const int src = n - (W - 1) + i;           // position within the step
        float x = 0.f;
        if (src >= 0) x = ldf(static_cast<const T*>(p.x) + static_cast<size_t>(t0 + src) * p.ldx + col);
        else if (resume) x = cs[W - 1 + src];
        cs[i] = x;
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) head_out_kernel(const MbHeadOut p) {
  const int V = p.vdim, lane = threadIdx.x & 31;
  const long long unit = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (unit >= static_cast<long long>(p.T) * p.heads) return;
  const size_t t = static_cast<size_t>(unit / p.heads);
  const int h = static_cast<int>(unit % p.heads);
  const float* o = p.o + unit * V;
  const T *gate = static_cast<const T*>(p.gate) + t * p.ld_gate + h * V, *w = static_cast<const T*>(p.norm_w) + h * p.w_stride;
  T* out = static_cast<T*>(p.out) + t * p.ld_out + h * V;
  float ss = 0.f;
  if (V <= 256 && V % 4 == 0 && p.ld_gate % 4 == 0 && p.ld_out % 4 == 0 &&
      ((reinterpret_cast<uintptr_t>(p.o) | reinterpret_cast<uintptr_t>(p.gate) | reinterpret_cast<uintptr_t>(p.norm_w) |
        reinterpret_cast<uintptr_t>(p.out)) & 15) == 0) {     // the head stays in registers
    float4 x[2], g[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int c = (lane + 32 * i) * 4;
      x[i] = c < V ? *reinterpret_cast<const float4*>(o + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      g[i] = c < V ? ld4(gate + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
    }
    const float inv = 1.f / sqrtf(warp_allsum(ss) / static_cast<float>(p.n) + p.eps);
    auto f = [&](float z) { return gate_of<T>(z, p.gate_silu, p.mult) * inv; };
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int c = (lane + 32 * i) * 4;
      if (c >= V) continue;
      const float4 a = ld4(w + c);
      st4(out + c, make_float4(x[i].x * a.x * f(g[i].x), x[i].y * a.y * f(g[i].y), x[i].z * a.z * f(g[i].z), x[i].w * a.w * f(g[i].w)));
    }
    return;
  }
  for (int c = lane; c < V; c += 32) ss = fmaf(o[c], o[c], ss);
  const float inv = 1.f / sqrtf(warp_allsum(ss) / static_cast<float>(p.n) + p.eps);
  for (int c = lane; c < V; c += 32) stf(out + c, o[c] * inv * ldf(w + c) * gate_of<T>(ldf(gate + c), p.gate_silu, p.mult));
}

template <typename T>
static int head_out(const MbHeadOut& p, cudaStream_t stream) {
  const long long units = static_cast<long long>(p.T) * p.heads;
  return launch_plain(head_out_kernel<T>, dim3(static_cast<unsigned>((units + 7) / 8)), dim3(256), 0, stream, p) == cudaSuccess
             ? MB_OK : MB_ERR_LAUNCH;
}

template <typename T, int RL4, int NC, bool HEADG>
static int scan_launch(const MbDelta& p, int warps, bool fuse, cudaStream_t stream) {
  constexpr int MAXT = RL4 <= 8 ? 512 : 256;
  const int cols = warps * 4 * NC, col_blocks = (p.vdim + cols - 1) / cols;
  const int per_token = ((HEADG ? 2 : 3) * 32 * RL4 + cols + (HEADG ? 4 : 2)) * 4;
  // tokens per stage: even, so that the second stage stays 16-byte aligned (a one-token step has no second stage)
  int chunk = p.one_token ? 1 : 40 * 1024 / (2 * per_token);
  if (!p.one_token) chunk = chunk > 16 ? 16 : chunk < 2 ? 2 : chunk & ~1;
  const size_t smem = static_cast<size_t>(2) * chunk * per_token + (fuse ? cols * 4 : 0) + 16;
  const dim3 grid(p.heads * col_blocks, p.B);
  if (fuse)
    return launch_plain(delta_scan_kernel<T, RL4, NC, MAXT, true, HEADG>, grid, dim3(warps * 32), smem, stream, p, col_blocks, chunk) ==
                   cudaSuccess ? MB_OK : MB_ERR_LAUNCH;
  if (launch_plain(delta_scan_kernel<T, RL4, NC, MAXT, false, HEADG>, grid, dim3(warps * 32), smem, stream, p, col_blocks, chunk) !=
      cudaSuccess)
    return MB_ERR_LAUNCH;
  const MbHeadOut o = {p.o, p.out, p.ld_out, p.gate, p.ld_gate, p.norm_w, p.T, p.heads, p.vdim, p.vdim, p.gate_silu, p.eps, p.out_mult};
  return head_out<T>(o, stream);
}

template <typename T, int RL4, bool HEADG>
static int scan_by_width(const MbDelta& p, int num_sms, cudaStream_t stream) {
  constexpr int max_warps = (RL4 <= 8 ? 512 : 256) / 32;
  const int head_warps = (p.vdim + 7) / 8;
  if (p.one_token && head_warps <= max_warps) return scan_launch<T, RL4, 2, HEADG>(p, head_warps, true, stream);
  // longer sequences: four columns per lane where the registers allow it (the rows are read once for all of them), and
  // CTAs of up to four warps as long as the grid has one per SM
  auto fit = [&](int per_warp) {
    const int hw = (p.vdim + per_warp - 1) / per_warp;
    int w = hw < 4 ? hw : 4;
    while (w > 1 && static_cast<long long>(p.B) * p.heads * ((hw + w - 1) / w) < num_sms) w >>= 1;
    return w;
  };
  if constexpr (RL4 <= 4) {
    if (p.vdim >= 16) return scan_launch<T, RL4, 4, HEADG>(p, fit(16), false, stream);
  }
  return scan_launch<T, RL4, 2, HEADG>(p, fit(8), false, stream);
}

template <typename T, int RL4>
static int scan(const MbDelta& p, int num_sms, cudaStream_t stream) {
  return p.z ? scan_by_width<T, RL4, false>(p, num_sms, stream) : scan_by_width<T, RL4, true>(p, num_sms, stream);
}

template <typename T>
static int run(const MbDelta& p, int num_sms, cudaStream_t stream) {
  const int vC = p.heads * p.vdim;
  const int units = p.kv_heads + decay_units(p) + (vC + 127) / 128;
  // vector loads: four channels per lane, every row and block start aligned to them
  const bool fast = p.dim <= 128 && p.dim % 4 == 0 && vC % 4 == 0 && p.taps >= 2 && p.taps <= 4 && p.ldx % 8 == 0 &&
                    p.q_off % 8 == 0 && p.k_off % 8 == 0 && p.v_off % 8 == 0 && (!p.z || p.ldz % 4 == 0) &&
                    ((reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.z) | reinterpret_cast<uintptr_t>(p.v) |
                      reinterpret_cast<uintptr_t>(p.dt_bias)) & 15) == 0;
  const int tile = p.T <= 4 * p.B ? 1 : 16;
  const dim3 grid((p.T + tile - 1) / tile, (units + 7) / 8);
  cudaError_t e;
  if (fast && p.taps == 4) e = launch_plain(delta_prep_fast_kernel<T, 4>, grid, dim3(256), 0, stream, p, tile);
  else if (fast && p.taps == 3) e = launch_plain(delta_prep_fast_kernel<T, 3>, grid, dim3(256), 0, stream, p, tile);
  else if (fast) e = launch_plain(delta_prep_fast_kernel<T, 2>, grid, dim3(256), 0, stream, p, tile);
  else e = launch_plain(delta_prep_kernel<T>, dim3(p.T, (units + 7) / 8), dim3(256), 0, stream, p);
  if (e != cudaSuccess) return MB_ERR_LAUNCH;
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

}  // namespace delta
}  // namespace mb

using namespace mb;

// Rows of the state per column: the smallest size the scan kernel is built for (0 = too large).
extern "C" int mb_delta_dim_pad(int dim) {
  const int sizes[] = {32, 64, 96, 128, 192, 256, 512};
  for (int s : sizes)
    if (dim <= s) return s;
  return 0;
}

extern "C" int mb_head_norm_gate(const MbHeadOut* p, int dtype, cudaStream_t stream) {
  if (p->T <= 0) return MB_OK;
  if (p->heads <= 0 || p->vdim <= 0 || p->n <= 0 || p->n > p->vdim) return MB_ERR_SHAPE;
  return dtype == kF32 ? delta::head_out<float>(*p, stream) : delta::head_out<__nv_bfloat16>(*p, stream);
}

extern "C" int mb_delta_rule(const MbDelta* p, int dtype, int num_sms, cudaStream_t stream) {
  if (p->T <= 0 || p->B <= 0) return MB_OK;
  if (p->heads <= 0 || p->kv_heads <= 0 || p->heads % p->kv_heads || p->dim <= 0 || p->vdim <= 0 || p->taps < 1 ||
      p->dim_pad != mb_delta_dim_pad(p->dim))
    return MB_ERR_SHAPE;
  if ((reinterpret_cast<uintptr_t>(p->q) | reinterpret_cast<uintptr_t>(p->k) | reinterpret_cast<uintptr_t>(p->g) |
       reinterpret_cast<uintptr_t>(p->state)) & 15)
    return MB_ERR_ALIGN;
  return dtype == kF32 ? delta::run<float>(*p, num_sms, stream) : delta::run<__nv_bfloat16>(*p, num_sms, stream);
}
