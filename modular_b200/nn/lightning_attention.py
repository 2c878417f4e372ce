"""Lightning attention: linear attention whose state decays by one constant per head.

Per head, with a state ``S`` [dim, vdim] kept in fp32: ``S <- decay S + k v^T``, ``o = S^T q``, where q, k and v are
projections behind a silu. The heads of a token, concatenated, are RMS-normed together, scaled by a weight and gated by
``sigmoid(W_g h)``. What a sequence carries between steps is ``S`` of every head, in the engine's state slots
(``state_shapes``), indexed by ``state_idx[s]`` (-1: start from zero and keep nothing) and read when the step continues a
sequence (``kv_len > q_len``).

On CUDA, ``csrc/kernels/lightning.cu``: bf16 prompts of heads up to 128 wide run in chunks on the tensor cores, everything
else token by token in fp32 arithmetic. CPU tensors take the token loop below.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .._native import lib as _lib
from .delta_rule import dim_pad, gemm_k, up8

CHUNK = 64             # tokens per step of the tensor-core kernel


@dataclass
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: tuple
    eps: float

    def __post_init__(self):
        if len(self.decay) != self.heads:
            raise ValueError(f"{len(self.decay)} decays for {self.heads} heads")

    @property
    def dim8(self) -> int:
        return up8(self.dim)

    @property
    def vdim8(self) -> int:
        return up8(self.vdim)

    def state_shapes(self) -> dict:
        return {"lightning": (self.heads, self.vdim8, dim_pad(self.dim8))}


class LightningAttention:
    """Weights of one mixer. ``w_in``: rows ``[q | k | v | gate]`` of a stacked input projection, heads padded to multiples
    of 8; ``w_o`` [width, heads * vdim8]."""

    def __init__(self, cfg: LightningConfig, tensors: dict, width_pad: int, device, dtype):
        c = self.cfg = cfg
        d, v = c.dim8, c.vdim8

        def rows(t, n, n_pad):
            t = t.view(c.heads, n, t.shape[1])
            return F.pad(t, (0, width_pad - t.shape[2], 0, n_pad - n)).reshape(-1, width_pad)

        self.w_in = torch.cat([rows(tensors["q"], c.dim, d), rows(tensors["k"], c.dim, d), rows(tensors["v"], c.vdim, v),
                               rows(tensors["g"], c.vdim, v)])
        self.k_off, self.v_off, self.g_off = c.heads * d, 2 * c.heads * d, c.heads * (2 * d + v)
        self.act_rows, self.in_rows = self.g_off, c.heads * (2 * d + 2 * v)     # silu covers q, k and v
        put = lambda t, dt=dtype: t.to(device=device, dtype=dt).contiguous()
        self.norm = put(F.pad(tensors["norm"].view(c.heads, c.vdim), (0, v - c.vdim)).reshape(-1))
        o = tensors["o"]
        o = F.pad(o.view(o.shape[0], c.heads, c.vdim), (0, v - c.vdim)).reshape(o.shape[0], -1)
        self.w_o = put(F.pad(o, (0, gemm_k(o.shape[1]) - o.shape[1], 0, width_pad - o.shape[0])))
        decay = torch.tensor(c.decay, dtype=torch.float64)
        self.decay = put(decay, torch.float32)
        self.decay_pow = put(decay.unsqueeze(1) ** torch.arange(CHUNK + 1, dtype=torch.float64), torch.float32)

    def __call__(self, x, state, state_idx, q_start, q_len, kv_len, one_token: bool):
        """x: this mixer's columns of the projection, q, k and v activated. Returns [T, columns of w_o]."""
        c, cols = self.cfg, self.cfg.heads * self.cfg.vdim8
        o = torch.empty(x.shape[0], self.w_o.shape[1], dtype=x.dtype, device=x.device)
        if o.shape[1] != cols:
            o[:, cols:].zero_()
        if x.is_cuda:
            _lib().lightning(x, 0, self.k_off, self.v_off, self.decay, self.decay_pow, o, state, state_idx, q_start, q_len, kv_len,
                             c.heads, c.dim8, c.vdim8, one_token)
            _lib().lightning_norm(o, x[:, self.g_off:], self.norm, cols, c.heads * c.vdim, c.eps)
            return o
        self.scan_reference(x, o, state, state_idx, q_start, q_len, kv_len)
        y = o[:, :cols].float()
        y = y * torch.rsqrt(y.pow(2).sum(-1, keepdim=True) / (c.heads * c.vdim) + c.eps) * self.norm.float()
        o[:, :cols] = (y * torch.sigmoid(x[:, self.g_off: self.g_off + cols].float())).to(o.dtype)
        return o

    def scan_reference(self, x, o, state, state_idx, q_start, q_len, kv_len):
        c, H, d, dv = self.cfg, self.cfg.heads, self.cfg.dim8, self.cfg.vdim8
        g = self.decay.view(H, 1, 1)
        for s in range(q_len.numel()):
            t0, n, slot = int(q_start[s]), int(q_len[s]), int(state_idx[s])
            rows = x[t0: t0 + n].float()
            q, k = rows[:, : H * d].view(n, H, d), rows[:, self.k_off: self.k_off + H * d].view(n, H, d)
            v = rows[:, self.v_off: self.v_off + H * dv].reshape(n, H, dv)
            S = state[slot, :, :, :d].clone() if slot >= 0 and int(kv_len[s]) > n else torch.zeros(H, dv, d)
            for t in range(n):
                S = g * S + v[t].unsqueeze(2) * k[t].unsqueeze(1)
                o[t0 + t, : H * dv] = torch.einsum("hvd,hd->hv", S, q[t]).reshape(-1).to(o.dtype)
            if slot >= 0:
                state[slot, :, :, :d] = S
                state[slot, :, :, d:] = 0
