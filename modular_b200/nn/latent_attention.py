"""Latent attention: queries and keys / values go through low-rank latents, and the cache keeps one row per token
(the normed key/value latent and a rotated key part that all heads share).

Runs in the absorbed form for prefill and decode alike: ``q_lat = W_uk^T q`` per head, attention over the cached rows,
``o = W_uv o_lat`` per head. Options: rotate-half or interleaved rotary pairs, a sliding window, a learned sink per head (a
score without key or value in the softmax denominator), a sigmoid output gate per value column or per head, and reading
another layer's cache rows (a layer without a key/value projection of its own).

Column layouts are padded for the kernels, with zeros: per head ``[dim -> multiple of 64 | rot_dim -> 64]`` for queries,
``[kv_rank -> a kernel size | rot_dim -> 64]`` for cache rows, vdim -> multiple of 8.

Kernels: ``mla_tc.cu`` (tcgen05: 512-wide latents, multiples of 128 heads), ``mla.cu`` (other sizes in bf16),
``mla_ragged.cu`` (fp32 and anything wider); CPU tensors take the PyTorch form.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from .._native import lib as _lib
from .delta_rule import gemm_k, pad_to, up8

_LATENT_SIZES = (64, 128, 192, 256, 384, 512)     # widths the tensor-core kernels are built for
_SPLIT_WS: dict = {}
_SPLIT_WS_BYTES = 64 << 20


def up64(n: int) -> int:
    return (n + 63) // 64 * 64


def latent_pad(kv_rank: int) -> int:
    return next((n for n in _LATENT_SIZES if kv_rank <= n), up64(kv_rank))


def rot_pad(rot_dim: int) -> int:
    return 64 if rot_dim <= 64 else up8(rot_dim)


@dataclass
class LatentAttentionConfig:
    heads: int
    dim: int                 # unrotated query / key width per head
    rot_dim: int             # width of the rotated part
    rot_dims: int            # how many of its values rotate (the first ones)
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rope_base: float
    eps: float
    own_cache: bool = True   # False: the layer reads another layer's cache rows
    interleaved: bool = False
    window: int = 0          # keys a query sees, itself included (0: all before it)
    sink: bool = True
    head_gate: bool = False  # the output gate is one number per head, applied inside the attention kernels

    @property
    def head_width(self) -> int:
        return up64(self.dim) + rot_pad(self.rot_dim)

    @property
    def cache_width(self) -> int:
        return latent_pad(self.kv_rank) + rot_pad(self.rot_dim)

    @property
    def vdim_pad(self) -> int:
        return up8(self.vdim)


def _split_ws(device) -> torch.Tensor:
    idx = device.index or 0
    if idx not in _SPLIT_WS:
        _SPLIT_WS[idx] = torch.empty(_SPLIT_WS_BYTES // 4, dtype=torch.float32, device=device)
    return _SPLIT_WS[idx]


def pad_heads(w: torch.Tensor, heads: int, rows: int, rows_pad: int) -> torch.Tensor:
    """[heads * rows, K] -> [heads * rows_pad, K] with zero rows after every head."""
    K = w.shape[1]
    if rows == rows_pad:
        return w
    out = torch.zeros(heads, rows_pad, K, dtype=w.dtype, device=w.device)
    out[:, :rows] = w.view(heads, rows, K)
    return out.view(heads * rows_pad, K)


class LatentAttention:
    """Weights of one mixer. ``w_in``: the projections that read the layer input, stacked ``[dq | dkv | g]`` (one GEMM)."""

    def __init__(self, cfg: LatentAttentionConfig, t: dict, width_pad: int, device, dtype):
        """``t``: the mixer's tensors by their short names (``dq``, ``dq.norm``, ``uk``, ``sink``, ...)."""
        c = self.cfg = cfg
        put = lambda x, dt=dtype: x.to(device=device, dtype=dt).contiguous()
        H, d, r, vp, Rp = c.heads, c.dim, c.rot_dim, c.vdim_pad, latent_pad(c.kv_rank)
        self.q_pad = gemm_k(c.q_rank)
        parts = [pad_to(t["dq"], self.q_pad, width_pad)]
        self.kv_off, at = -1, self.q_pad
        if c.own_cache:
            n = c.kv_rank + r
            parts.append(pad_to(t["dkv"], up8(n), width_pad))
            self.kv_off, at = at, at + up8(n)
        self.g_off = at
        parts.append(pad_to(t["g"], up8(H), width_pad) if c.head_gate else pad_to(pad_heads(t["g"], H, c.vdim, vp), H * vp, width_pad))
        self.w_in = put(torch.cat(parts))
        self.q_norm = put(t["dq.norm"])
        self.kv_norm = put(t["dkv.norm"]) if c.own_cache else None
        uq = t["uq"].view(H, d + r, c.q_rank)
        new = lambda *s: torch.zeros(*s, dtype=uq.dtype, device=uq.device)
        q = new(H, c.head_width, self.q_pad)
        q[:, :d, : c.q_rank] = uq[:, :d]
        q[:, up64(d): up64(d) + r, : c.q_rank] = uq[:, d:]
        self.w_uq = put(q.view(H * c.head_width, self.q_pad))
        uk = new(H, Rp, up64(d))
        uk[:, : c.kv_rank, :d] = t["uk"].view(H, d, c.kv_rank).transpose(1, 2)
        self.w_uk = put(uk)                                          # [h, latent, dim]: queries into latent space
        uv = new(H, vp, Rp)
        uv[:, : c.vdim, : c.kv_rank] = t["uv"].view(H, c.vdim, c.kv_rank)
        self.w_uv = put(uv)                                          # [h, vdim, latent]: latent outputs to values
        self.sink = put(t["sink"], torch.float32) if c.sink else None
        self.w_o = put(pad_to(pad_heads(t["o"].t().contiguous(), H, c.vdim, vp).t(), width_pad, gemm_k(H * vp)))

    def __call__(self, x, lin, cache, cos_sin, positions, slots, block_table, q_start, q_len, kv_len, one_token: bool):
        """x [T, width] -> [T, width]; ``cache`` [pages, page, >= cache_width] is this layer's (or the shared) plane."""
        c, T = self.cfg, x.shape[0]
        H, dp, Dp, Rp = c.heads, up64(c.dim), rot_pad(c.rot_dim), latent_pad(c.kv_rank)
        px = lin(x, self.w_in)
        c_q = torch.empty(T, self.q_pad, dtype=x.dtype, device=x.device)
        latent_post_down(self, px, c_q, positions, cos_sin, slots, cache)
        q = lin(c_q, self.w_uq)                                      # [T, h * (dim | rotated)]
        rotate_heads(q[:, dp:], H, c.head_width, c.rot_dims, c.interleaved, positions, cos_sin)
        q_lat = torch.empty(T, H * Rp, dtype=x.dtype, device=x.device)
        ops.batched_linear_heads(q, self.w_uk, q_lat, c.head_width, Rp)
        q_rope = q.view(T, H, c.head_width)[:, :, dp:]
        o_lat = latent_attention(q_lat.view(T, H, Rp), q_rope, cache, block_table, q_start, q_len, kv_len, c.scale, self.sink,
                                 one_token, c.window, px[:, self.g_off: self.g_off + H] if c.head_gate else None)
        width = H * c.vdim_pad
        o = torch.empty(T, self.w_o.shape[1], dtype=x.dtype, device=x.device)
        if o.shape[1] != width:
            o[:, width:].zero_()
        ops.batched_linear_heads(o_lat.view(T, H * Rp), self.w_uv, o, Rp, c.vdim_pad)
        if not c.head_gate:
            ops.sigmoid_gate(o, px[:, self.g_off:], width)
        return lin(o, self.w_o)


def latent_post_down(m: LatentAttention, px, c_q, positions, cos_sin, slots, cache):
    """Query latent normed into ``c_q``; key/value latent normed and its rotated part stored in the tokens' cache rows."""
    c = m.cfg
    Rp, Dp = latent_pad(c.kv_rank), rot_pad(c.rot_dim)
    if px.is_cuda:
        _lib().latent_post_down(px, c.q_rank, m.q_norm, c_q, m.kv_off, c.kv_rank, Rp, m.kv_norm, c.rot_dim, Dp, c.rot_dims,
                                c.interleaved, c.eps, positions, cos_sin, slots, cache if c.own_cache else None)
        return
    rms = lambda t, w: t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + c.eps) * w.float()
    c_q.zero_()
    c_q[:, : c.q_rank] = rms(px[:, : c.q_rank].float(), m.q_norm).to(c_q.dtype)
    if not c.own_cache:
        return
    kv = px[:, m.kv_off: m.kv_off + c.kv_rank + c.rot_dim].float()
    rows = torch.zeros(px.shape[0], Rp + Dp)
    rows[:, : c.kv_rank] = rms(kv[:, : c.kv_rank], m.kv_norm)
    rows[:, Rp: Rp + c.rot_dim] = kv[:, c.kv_rank:]
    rotate_heads(rows[:, Rp:], 1, Dp, c.rot_dims, c.interleaved, positions, cos_sin)
    page = cache.shape[1]
    ok = slots >= 0
    cache[slots[ok] // page, slots[ok] % page, : Rp + Dp] = rows[ok].to(cache.dtype)


def rotate_heads(x, heads, head_stride, dims, interleaved, positions, cos_sin):
    """In place: the first ``dims`` values of every head of ``x`` (head i starts at column ``i * head_stride``)."""
    if x.is_cuda:
        _lib().rotate_heads(x, heads, head_stride, dims, interleaved, positions, cos_sin)
        return
    cs = cos_sin[positions.long()]
    cos, sin = cs[:, : dims // 2], cs[:, dims // 2:]
    for h in range(heads):
        part = x[:, h * head_stride: h * head_stride + dims]
        part.copy_(ops.reference.apply_rope(part.unsqueeze(1), cos, sin, interleaved).squeeze(1))


def latent_attention(q_lat, q_rope, cache, block_table, q_start, q_len, kv_len, scale, sink=None, one_token=False, window=0, gate=None):
    """Absorbed attention over paged latent rows; returns [T, h, latent]. ``gate`` [T, h]: heads are multiplied by its sigmoid."""
    if q_lat.is_cuda:
        out = torch.empty_like(q_lat)
        if q_lat.dtype == torch.bfloat16:
            ops.ensure_mla_split_workspace(q_lat.device)
        _lib().latent_attention(q_lat, q_rope, cache, block_table, q_start, q_len, kv_len, out, scale, sink, one_token,
                                _split_ws(q_lat.device), window=window, gate=gate)
        return out
    T, H, Rp = q_lat.shape
    LD, page = Rp + q_rope.shape[2], cache.shape[1]
    out = torch.zeros_like(q_lat)
    q = torch.cat([q_lat, q_rope], -1).float()
    for s in range(q_len.numel()):
        t0, n, kl = int(q_start[s]), int(q_len[s]), int(kv_len[s])
        k = cache[block_table[s, : (kl + page - 1) // page].long()].reshape(-1, cache.shape[2])[:kl, :LD].float()
        sc = torch.einsum("qhd,kd->hqk", q[t0: t0 + n], k) * scale
        dist = torch.arange(n).unsqueeze(1) + (kl - n) - torch.arange(kl).unsqueeze(0)
        sc = sc.masked_fill((dist < 0) | (dist >= (window or kl)), float("-inf"))
        if sink is not None:
            sc = torch.cat([sc, sink.view(H, 1, 1).expand(H, n, 1)], -1)
        p = torch.softmax(sc, -1)[..., :kl]
        o = torch.einsum("hqk,kd->qhd", p, k[:, :Rp])
        if gate is not None:
            o = o * torch.sigmoid(gate[t0: t0 + n].float()).unsqueeze(2)
        out[t0: t0 + n] = o.to(out.dtype)
    return out
