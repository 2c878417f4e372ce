"""Generalized delta rule: linear attention whose state decays by a factor per key channel and forgets, at a rate per key channel, what
it holds under the current key.

Per head, with a state ``S`` [dim, vdim] kept in fp32 and ``u`` the unit vector of the key ``k``:

    S <- (diag(w) - (a * u) u^T) S + k v^T;    o = S^T r

where both terms of the transition read the old state, ``w = exp(-exp(-1/2) sigmoid(W_w2 tanh(W_w1 h) + w0))`` and
``a = sigmoid(W_a h + b)`` per key channel. Every head's output is RMS-normed, scaled by a weight of its own and gated by
``sigmoid(W_g h)``. What a sequence carries between steps is ``S`` of every head, in the engine's state slots (``state_shapes``),
indexed by ``state_idx[s]`` (-1: start from zero and keep nothing) and read when the step continues a sequence (``kv_len > q_len``).

Heads are padded to multiples of 8 in the weights, with zeros. On CUDA, ``csrc/kernels/general_delta.cu``; CPU tensors take the
token loop below.
"""

from __future__ import annotations

import math
from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .. import ops
from .._native import lib as _lib
from .delta_rule import dim_pad, gemm_k, pad_to, up8


@dataclass
class GeneralDeltaConfig:
    heads: int
    dim: int                 # of keys and values
    rank: int                # of the decay projection
    eps: float

    @property
    def dim8(self) -> int:
        return up8(self.dim)

    def state_shapes(self) -> dict:
        return {"gdelta": (self.heads, self.dim8, dim_pad(self.dim8))}


class GeneralDelta:
    """Weights of one mixer. ``w_in``: the projections that read the layer input, stacked ``[r | k | v | g | a | w1]`` (one GEMM);
    ``w_w2`` the second half of the decay projection; ``w_o`` [width, heads * dim8]."""

    def __init__(self, cfg: GeneralDeltaConfig, t: dict, width_pad: int, device, dtype):
        """``t``: the mixer's tensors by their short names (``r``, ``w1``, ``a.b``, ...)."""
        c = self.cfg = cfg
        H, d = c.heads, c.dim8
        put = lambda x, dt=dtype: x.to(device=device, dtype=dt).contiguous()
        heads = lambda w, cols: F.pad(w.view(H, c.dim, w.shape[1]), (0, cols - w.shape[1], 0, d - c.dim)).reshape(H * d, cols)
        vector = lambda v, dt: put(F.pad(v.view(H, c.dim), (0, d - c.dim)).reshape(-1), dt)
        self.rank_pad = gemm_k(c.rank)
        self.w_in = put(torch.cat([heads(t[n], width_pad) for n in ("r", "k", "v", "g", "a")] + [pad_to(t["w1"], self.rank_pad, width_pad)]))
        self.k_off, self.v_off, self.g_off, self.a_off, self.w_off = (i * H * d for i in range(1, 6))
        self.w_w2 = put(heads(t["w2"], self.rank_pad))
        self.w_bias, self.a_bias = vector(t["w0"], torch.float32), vector(t["a.b"], torch.float32)
        self.norm = vector(t["norm"], dtype)
        o = t["o"]
        self.w_o = put(pad_to(F.pad(o.view(o.shape[0], H, c.dim), (0, d - c.dim)).reshape(o.shape[0], -1), width_pad, gemm_k(H * d)))

    def __call__(self, x, lin, state, state_idx, q_start, q_len, kv_len, one_token: bool):
        """x [T, width] -> [T, width]; ``lin`` is the GEMM for this step's size."""
        c, cols = self.cfg, self.cfg.heads * self.cfg.dim8
        px = lin(x, self.w_in)
        z = ops.linear(ops.tanh(px[:, self.w_off: self.w_off + self.rank_pad]), self.w_w2, out_dtype=torch.float32)
        out = torch.empty(x.shape[0], self.w_o.shape[1], dtype=x.dtype, device=x.device)
        if out.shape[1] != cols:
            out[:, cols:].zero_()
        self.mix(px, z, out, state, state_idx, q_start, q_len, kv_len, one_token)
        return lin(out, self.w_o)

    def mix(self, px, z, out, state, state_idx, q_start, q_len, kv_len, one_token: bool):
        """From the stacked projection and the decay logits ``z`` (fp32) to the gated heads in ``out``."""
        c, T = self.cfg, px.shape[0]
        if not px.is_cuda:
            return self.scan_reference(px, z, out, state, state_idx, q_start, q_len, kv_len)
        f32 = lambda n: torch.empty(n, dtype=torch.float32, device=px.device)
        fused = one_token and c.dim8 <= 128                  # one launch, no scratch
        _lib().general_delta(px, 0, self.k_off, self.v_off, self.a_off, self.a_bias, z, self.w_bias, px[:, self.g_off: self.a_off], self.norm,
                             c.eps, c.dim, f32(0 if fused else T * c.heads * (4 * dim_pad(c.dim8) + 4)),
                             f32(0 if fused else T * c.heads * c.dim8), out, state, state_idx, q_start, q_len, kv_len, c.heads, c.dim8,
                             c.dim8, one_token)

    def scan_reference(self, px, z, out, state, state_idx, q_start, q_len, kv_len):
        c, H, d = self.cfg, self.cfg.heads, self.cfg.dim8
        decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(z + self.w_bias)).view(-1, H, d)
        rate = torch.sigmoid(px[:, self.a_off: self.w_off].float() + self.a_bias).view(-1, H, d)
        for s in range(q_len.numel()):
            t0, n, slot = int(q_start[s]), int(q_len[s]), int(state_idx[s])
            rows = px[t0: t0 + n].float()
            r, k, v, g = (rows[:, i * H * d: (i + 1) * H * d].reshape(n, H, d) for i in range(4))
            u = k / torch.sqrt(k.pow(2).sum(-1, keepdim=True) + 1e-6)
            S = state[slot, :, :, :d].clone() if slot >= 0 and int(kv_len[s]) > n else torch.zeros(H, d, d)      # [head, column, row]
            o = torch.empty(n, H, d)
            for t in range(n):
                held = torch.einsum("hvd,hd->hv", S, u[t])
                S = S * decay[t0 + t].unsqueeze(1) + v[t].unsqueeze(2) * k[t].unsqueeze(1)
                S = S - held.unsqueeze(2) * (rate[t0 + t] * u[t]).unsqueeze(1)
                o[t] = torch.einsum("hvd,hd->hv", S, r[t])
            if slot >= 0:
                state[slot, :, :, :d] = S
            o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / c.dim + c.eps)
            out[t0: t0 + n, : H * d] = (o.reshape(n, -1) * self.norm.float() * torch.sigmoid(g.reshape(n, -1))).to(out.dtype)
