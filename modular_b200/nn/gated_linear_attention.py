"""Gated linear attention: linear attention whose state decays by a factor per key channel that depends on the token.

Per head, with a state ``S`` [dim, vdim] kept in fp32: ``S <- diag(alpha) S + k v^T``, ``o = S^T q``, with
``alpha = sigmoid(W_a2 W_a1 h + b)^(1 / tau)`` and ``q`` scaled by ``dim^(-1/2)``. Every head's output is RMS-normed, scaled by a
weight and gated by ``silu(W_g h)``. What a sequence carries between steps is ``S`` of every head, in the engine's state slots
(``state_shapes``), indexed by ``state_idx[s]`` (-1: start from zero and keep nothing) and read when the step continues a
sequence (``kv_len > q_len``).

Heads are padded to multiples of 8 in the weights, with zeros. On CUDA, ``csrc/kernels/gla.cu``; CPU tensors take the token
loop below.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .. import ops
from .._native import lib as _lib
from .delta_rule import dim_pad, gemm_k, pad_to, up8


@dataclass
class GatedLinearConfig:
    heads: int
    dim: int
    vdim: int
    rank: int                # of the decay projection
    tau: float
    eps: float

    @property
    def dim8(self) -> int:
        return up8(self.dim)

    @property
    def vdim8(self) -> int:
        return up8(self.vdim)

    def state_shapes(self) -> dict:
        return {"gla": (self.heads, self.vdim8, dim_pad(self.dim8))}


class GatedLinearAttention:
    """Weights of one mixer. ``w_in``: the projections that read the layer input, stacked ``[q | k | v | g | a1]`` (one GEMM);
    ``w_a2`` the second half of the decay projection; ``w_o`` [width, heads * vdim8]."""

    def __init__(self, cfg: GatedLinearConfig, t: dict, width_pad: int, device, dtype):
        """``t``: the mixer's tensors by their short names (``q``, ``a1``, ``a2.b``, ...)."""
        c = self.cfg = cfg
        H, d, v = c.heads, c.dim8, c.vdim8
        put = lambda x, dt=dtype: x.to(device=device, dtype=dt).contiguous()

        def heads(w, n, n_pad, cols):
            return F.pad(w.view(H, n, w.shape[1]), (0, cols - w.shape[1], 0, n_pad - n)).reshape(H * n_pad, cols)

        self.rank_pad = gemm_k(c.rank)
        self.w_in = put(torch.cat([heads(t["q"], c.dim, d, width_pad), heads(t["k"], c.dim, d, width_pad), heads(t["v"], c.vdim, v, width_pad),
                                   heads(t["g"], c.vdim, v, width_pad), pad_to(t["a1"], self.rank_pad, width_pad)]))
        self.k_off, self.v_off, self.g_off, self.a_off = H * d, 2 * H * d, H * (2 * d + v), H * (2 * d + 2 * v)
        self.w_a2 = put(heads(t["a2"], c.dim, d, self.rank_pad))
        self.a_bias = put(F.pad(t["a2.b"].view(H, c.dim), (0, d - c.dim)).reshape(-1), torch.float32)
        self.norm = put(F.pad(t["norm"], (0, v - c.vdim)))
        o = t["o"]
        self.w_o = put(pad_to(F.pad(o.view(o.shape[0], H, c.vdim), (0, v - c.vdim)).reshape(o.shape[0], -1), width_pad, gemm_k(H * v)))

    def __call__(self, x, lin, state, state_idx, q_start, q_len, kv_len, one_token: bool):
        """x [T, width] -> [T, width]; ``lin`` is the GEMM for this step's size."""
        c, T, cols = self.cfg, x.shape[0], self.cfg.heads * self.cfg.vdim8
        px = lin(x, self.w_in)
        z = ops.linear(px[:, self.a_off: self.a_off + self.rank_pad], self.w_a2, out_dtype=torch.float32)
        out = torch.empty(T, self.w_o.shape[1], dtype=x.dtype, device=x.device)
        if out.shape[1] != cols:
            out[:, cols:].zero_()
        self.mix(px, z, out, state, state_idx, q_start, q_len, kv_len, one_token)
        return lin(out, self.w_o)

    def mix(self, px, z, out, state, state_idx, q_start, q_len, kv_len, one_token: bool):
        """From the stacked projection and the decay logits ``z`` (fp32) to the gated heads in ``out``."""
        c = self.cfg
        if not px.is_cuda:
            return self.scan_reference(px, z, out, state, state_idx, q_start, q_len, kv_len)
        o = torch.empty(px.shape[0], c.heads * c.vdim8, dtype=torch.float32, device=px.device)
        _lib().gla(px, 0, self.k_off, self.v_off, z, self.a_bias, c.dim ** -0.5, 1.0 / c.tau, px[:, self.g_off: self.a_off], True, 1.0,
                   self.norm, c.eps, c.vdim, o, out, state, state_idx, q_start, q_len, kv_len, c.heads, c.dim8, c.vdim8, one_token)

    def scan_reference(self, px, z, out, state, state_idx, q_start, q_len, kv_len):
        c, H, d, dv = self.cfg, self.cfg.heads, self.cfg.dim8, self.cfg.vdim8
        alpha = torch.exp(F.logsigmoid(z + self.a_bias) / c.tau)
        for s in range(q_len.numel()):
            t0, n, slot = int(q_start[s]), int(q_len[s]), int(state_idx[s])
            rows = px[t0: t0 + n].float()
            q, k = rows[:, : H * d].view(n, H, d) * c.dim ** -0.5, rows[:, self.k_off: self.v_off].view(n, H, d)
            v, g = rows[:, self.v_off: self.g_off].reshape(n, H, dv), alpha[t0: t0 + n].view(n, H, 1, d)
            S = state[slot, :, :, :d].clone() if slot >= 0 and int(kv_len[s]) > n else torch.zeros(H, dv, d)
            o = torch.empty(n, H, dv)
            for t in range(n):
                S = g[t] * S + v[t].unsqueeze(2) * k[t].unsqueeze(1)
                o[t] = torch.einsum("hvd,hd->hv", S, q[t])
            if slot >= 0:
                state[slot, :, :, :d] = S
                state[slot, :, :, d:] = 0
            o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / c.vdim + c.eps) * self.norm.float()
            out[t0: t0 + n, : H * dv] = (o.reshape(n, -1) * F.silu(rows[:, self.g_off: self.a_off])).to(out.dtype)
