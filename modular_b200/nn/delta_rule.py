"""Gated delta rule with a decay per key channel or per head, behind short convolutions (a linear-attention mixer).

Per head, with a state ``S`` [dim, vdim] kept in fp32:

    S <- diag(g) S;    u = beta (v - S^T k);    S <- S + k u^T;    o = S^T q

q, k, v are projections that pass a causal depthwise convolution and silu, q and k are unit vectors, the decay is
``g = exp(-exp(A_log) softplus(a + dt_bias))`` with ``a = W_a2 W_a1 h`` per channel or ``a = W_a h`` per head, and the output is
RMS-normed per head, scaled and gated by ``sigmoid(W_g2 W_g1 h)`` or ``silu(W_g h)``. What a sequence carries between steps is ``S`` of every head and the last ``taps - 1`` inputs
of the convolutions: two tensors of the engine's state slots (``state_specs``), indexed by ``state_idx[s]`` (-1: start
from zero and keep nothing), read when the step continues a sequence (``kv_len > q_len``).

On CUDA, bf16 and fp32 run ``csrc/kernels/delta_rule.cu``; CPU tensors take the token loop below.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .. import ops
from .._native import lib as _lib

_PAD = (32, 64, 96, 128, 192, 256, 512)      # key widths the scan kernel is built for


def dim_pad(dim: int) -> int:
    """Rows per state column: the key width rounded up to one the scan kernel is built for."""
    for n in _PAD:
        if dim <= n:
            return n
    raise ValueError(f"key width {dim} is beyond the largest supported one ({_PAD[-1]})")


def up8(n: int) -> int:
    return (n + 7) // 8 * 8


def gemm_k(n: int) -> int:
    """A GEMM's inner width: a multiple of 8, at least one 64-wide block."""
    return max(64, up8(n))


def pad_to(w: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    """``w`` with zero rows and columns appended."""
    return F.pad(w, (0, cols - w.shape[1], 0, rows - w.shape[0])) if (rows, cols) != tuple(w.shape) else w


@dataclass
class DeltaRuleConfig:
    hidden: int
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int              # low-rank decays per channel and gates behind a sigmoid, or, with head_decay,
    gate_rank: int               # one decay per head and a full-rank gate behind silu (both ranks unused)
    eps: float
    head_decay: bool = False
    out_mult: float = 1.0        # factor on the output

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def blocks(self) -> tuple:
        """(name, rows, first row) of the stacked input projection; every block starts at a multiple of 8 (the
        low-rank ones, which are GEMM inputs, are at least 64 wide)."""
        out, at = [], 0
        tail = ((("g", self.heads * self.vdim), ("a", self.heads)) if self.head_decay else
                (("a1", self.decay_rank), ("g1", self.gate_rank)))
        for name, n in (("q", self.kv_heads * self.dim), ("k", self.kv_heads * self.dim), ("v", self.heads * self.vdim),
                        *tail, ("b", self.heads)):
            out.append((name, n, at))
            at += self.block_rows(name, n)
        return tuple(out)

    @staticmethod
    def block_rows(name: str, n: int) -> int:
        return gemm_k(n) if name in ("a1", "g1") else up8(n)

    def state_shapes(self) -> dict:
        return {"delta": (self.heads, self.vdim, dim_pad(self.dim)), "conv": (self.channels, self.taps - 1)}


def delta_step_reference(q, k, v, g, beta, S):
    """One token of one sequence: q, k, g [H, d], v [H, dv], beta [H], S [H, dv, d] (updated in place); returns o [H, dv]."""
    S *= g.unsqueeze(1)
    u = beta.unsqueeze(-1) * (v - torch.einsum("hvd,hd->hv", S, k))
    S += u.unsqueeze(-1) * k.unsqueeze(1)
    return torch.einsum("hvd,hd->hv", S, q)


class DeltaRule:
    """Weights of one mixer. ``w_in``: the projections that read the layer input, stacked ``[q | k | v | a1 | g1 | b]`` or
    ``[q | k | v | g | a | b]`` (one GEMM); ``w_a2`` / ``w_g2``: the second halves of low-rank decay and gate projections; ``w_o``."""

    def __init__(self, cfg: DeltaRuleConfig, tensors: dict, width_pad: int, device, dtype):
        """``tensors``: the mixer's tensors by their short names (``q``, ``q.conv``, ``a1``, ...)."""
        c = self.cfg = cfg
        put = lambda t, dt=dtype: t.to(device=device, dtype=dt).contiguous()
        self.w_in = put(torch.cat([pad_to(tensors[n], c.block_rows(n, rows), width_pad) for n, rows, _ in c.blocks]))
        self.off = {n: at for n, _, at in c.blocks}
        self.in_rows = self.w_in.shape[0]
        self.conv_w = put(torch.cat([tensors[n + ".conv"] for n in "qkv"]))
        if not c.head_decay:
            self.w_a2 = put(pad_to(tensors["a2"], up8(c.heads * c.dim), c.block_rows("a1", c.decay_rank)))
            self.w_g2 = put(pad_to(tensors["g2"], up8(c.heads * c.vdim), c.block_rows("g1", c.gate_rank)))
        self.A_log = put(tensors["A_log"], torch.float32)
        self.dt_bias = put(tensors["dt_bias"], torch.float32)
        self.norm = put(tensors["norm"])
        self.w_o = put(pad_to(tensors["o"], width_pad, gemm_k(c.heads * c.vdim)))

    def __call__(self, x, lin, state, conv_state, state_idx, q_start, q_len, kv_len, one_token: bool):
        """x [T, width] -> [T, width]; ``lin`` is the GEMM for this step's size."""
        c, T, dev = self.cfg, x.shape[0], x.device
        px = lin(x, self.w_in)
        width = self.w_o.shape[1]
        out = torch.empty(T, width, dtype=x.dtype, device=dev)
        if width != c.heads * c.vdim:
            out[:, c.heads * c.vdim:].zero_()
        self.mix(px, out, state, conv_state, state_idx, q_start, q_len, kv_len, one_token)
        return lin(out, self.w_o)

    def mix(self, px, out, state, conv_state, state_idx, q_start, q_len, kv_len, one_token: bool):
        """From the stacked projection ``px`` to the gated heads, in the first heads * vdim columns of ``out``."""
        c = self.cfg
        if c.head_decay:
            z, gate = None, px[:, self.off["g"]: self.off["g"] + c.heads * c.vdim]
        else:
            a0, g0 = self.off["a1"], self.off["g1"]
            z = ops.linear(px[:, a0: a0 + self.w_a2.shape[1]], self.w_a2, out_dtype=torch.float32)
            gate = ops.linear(px[:, g0: g0 + self.w_g2.shape[1]], self.w_g2)
        core = delta_rule_cuda if px.is_cuda else delta_rule_reference
        core(self, px, z, gate, out, state, conv_state, state_idx, q_start, q_len, kv_len, one_token)


def delta_rule_cuda(m: DeltaRule, px, z, gate, out, state, conv_state, state_idx, q_start, q_len, kv_len, one_token):
    c, T = m.cfg, px.shape[0]
    dp = dim_pad(c.dim)
    sizes = (T * c.kv_heads * dp, T * c.kv_heads * dp, T * c.heads * (1 if c.head_decay else dp), T * c.heads * c.vdim, T * c.heads, T * c.kv_heads,
             T * c.heads * c.vdim)
    ends, at = [], 0
    for n in sizes:                       # one allocation, every part 16-byte aligned
        ends.append((at, n))
        at += (n + 3) // 4 * 4
    buf = torch.empty(at, dtype=torch.float32, device=px.device)
    _lib().delta_rule(px, m.off["q"], m.off["k"], m.off["v"], m.off["b"], m.conv_w, z, m.A_log, m.dt_bias, gate, m.norm, c.eps,
                      [buf[s: s + n] for s, n in ends], out, state, conv_state, state_idx, q_start, q_len, kv_len, c.heads,
                      c.kv_heads, c.dim, c.vdim, one_token, a_off=m.off.get("a", -1), gate_silu=c.head_decay, out_mult=c.out_mult)


def delta_rule_reference(m: DeltaRule, px, z, gate, out, state, conv_state, state_idx, q_start, q_len, kv_len, one_token=False):
    c = m.cfg
    H, KH, d, dv, W = c.heads, c.kv_heads, c.dim, c.vdim, c.taps
    raw = torch.cat([px[:, m.off[n]: m.off[n] + r].float() for n, r, _ in c.blocks[:3]], 1)
    beta = torch.sigmoid(px[:, m.off["b"]: m.off["b"] + H].float())
    a = px[:, m.off["a"]: m.off["a"] + H] if c.head_decay else z[:, : H * d]
    g = torch.exp(-torch.exp(m.A_log).view(1, H, 1) * F.softplus(a.float() + m.dt_bias).view(a.shape[0], H, -1))
    rep = H // KH
    unit = lambda t: t / torch.sqrt((t * t).sum(-1, keepdim=True) + 1e-6)
    for s in range(q_len.numel()):
        t0, n, slot = int(q_start[s]), int(q_len[s]), int(state_idx[s])
        resume = slot >= 0 and int(kv_len[s]) > n
        hist = conv_state[slot].t() if resume and W > 1 else torch.zeros(W - 1, c.channels)
        seq = torch.cat([hist, raw[t0: t0 + n]], 0)
        y = F.silu(sum(seq[j: j + n] * m.conv_w[:, j].float() for j in range(W)))
        if slot >= 0 and W > 1:
            conv_state[slot] = seq[seq.shape[0] - (W - 1):].t()
        q, k, v = y.split([KH * d, KH * d, H * dv], 1)
        q = (unit(q.reshape(n, KH, d)) / d ** 0.5).repeat_interleave(rep, 1)
        k = unit(k.reshape(n, KH, d)).repeat_interleave(rep, 1)
        v = v.reshape(n, H, dv)
        S = state[slot, :, :, :d].clone() if resume else torch.zeros(H, dv, d)
        o = torch.stack([delta_step_reference(q[t], k[t], v[t], g[t0 + t], beta[t0 + t], S) for t in range(n)])
        if slot >= 0:
            state[slot, :, :, :d] = S
        o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + c.eps) * m.norm.float()
        act = F.silu if c.head_decay else torch.sigmoid
        o = o.reshape(n, H * dv) * act(gate[t0: t0 + n, : H * dv].float()) * c.out_mult
        out[t0: t0 + n, : H * dv] = o.to(out.dtype)
