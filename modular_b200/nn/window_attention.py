"""Softmax attention over the keys of a sliding window, with grouped heads, partial rotation, a sink, and optionally biases, normed
queries and keys and an output gate per head.

A query at position i sees the keys j with ``0 <= i - j < window`` (0: all before it). Queries and keys rotate in
neighbouring pairs (or pairs half the rotated width apart, ``halves``) over their first ``rot_dims`` dimensions; ``qk_norm``
RMS-norms every head of both before that. ``bias`` adds a vector to q, k and v (in fp32, on the way through the rotation). ``sink`` is one score per query head that takes part in the softmax denominator
only: ``p_j = exp(s_j) / (exp(sink) + sum_j exp(s_j))``. ``head_gate`` multiplies a head's output by ``sigmoid(W_g h)``, inside
the attention kernels; ``out_mult`` is a further factor on it.

The cache is the paged key/value cache of the grouped-query families ``[pages, 2, planes, kv heads, page, head width]``.
Keys and values share one head width, zero-padded: 64 or 128 where the tensor-core kernels fit (``head_width``), and the
query heads of a group are padded to a power of two; both paddings live in the weights, so no kernel ever copies rows.

On CUDA, bf16 with such heads runs ``csrc/kernels/attention_tc.cu`` (prompts, tcgen05) and ``attention_tma.cu`` (decode steps;
prompts of 64-wide heads); fp32 and other sizes run ``attention_window.cu``. CPU tensors take the PyTorch forms below.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from .. import ops
from .._native import lib as _lib
from .delta_rule import up8
from .rotary_embedding import RopeScaling

MAX_GROUP = 16         # query heads per key/value head of the tensor-core kernels


def head_width(widest: int) -> int:
    """Columns of a head in projections and cache: one of the tensor-core widths, or a multiple of 8 beyond them."""
    return 64 if widest <= 64 else 128 if widest <= 128 else up8(widest)


@dataclass
class WindowAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int = 0
    rope_base: float = 10000.0
    rope_scaling: Optional[RopeScaling] = None
    window: int = 0                  # 0: every key before the query
    zero_sink: bool = False          # a sink of score 0 for every head
    sink: bool = False               # a learned sink
    halves: bool = False             # pairs (i, i + rot_dims / 2)
    bias: bool = False               # on q, k and v; needs halves
    qk_norm: bool = False
    eps: float = 1e-6                # of those norms
    head_gate: bool = False
    out_mult: float = 1.0            # needs head_gate

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} heads are no multiple of {self.kv_heads} key/value heads")
        if self.rot_dims % 2 or self.rot_dims > self.dim:
            raise ValueError(f"{self.rot_dims} rotated dimensions of {self.dim}")
        if self.bias and not self.halves:
            raise ValueError("biases are added by the kernel for pairs half the rotated width apart")
        if self.out_mult != 1.0 and not self.head_gate:
            raise ValueError("a factor on the output is part of the head gate")
        if self.window < 0:
            raise ValueError("a window holds at least the token itself")

    @property
    def group_pad(self) -> int:
        """Query heads per key/value head, padded to a power of two where the tensor-core kernels apply."""
        g = self.heads // self.kv_heads
        return 1 << (g - 1).bit_length() if g <= MAX_GROUP and head_width(max(self.dim, self.vdim)) <= 128 else g

    @property
    def heads_pad(self) -> int:
        return self.kv_heads * self.group_pad


@dataclass
class AttentionPlan:
    """Work split of one step for the tensor-core kernels: prompt tiles, or one row per sequence."""
    tile_seq: Optional[torch.Tensor] = None
    tile_q0: Optional[torch.Tensor] = None
    decode_seq: Optional[torch.Tensor] = None


def tensor_core_plan(group: int, hd: int, dtype, page: int, q_start, q_len, T: int, one_token: bool) -> Optional[AttentionPlan]:
    """The plan of a step for heads in groups of ``group``, or None where the CUDA-core kernel runs."""
    if not q_len.is_cuda or dtype != torch.bfloat16 or hd not in (64, 128) or page % 64 or group > MAX_GROUP or group & (group - 1):
        return None
    if one_token:
        ops.ensure_attention_split_workspace(q_len.device)
        return AttentionPlan(decode_seq=q_start)       # row i is sequence i
    tok = (128 if hd == 128 else 64) // group
    n = T // tok + q_len.numel()
    tiles = torch.empty(2, n, dtype=torch.int32, device=q_len.device)
    _lib().attention_plan(q_len, tok, tiles[0], tiles[1])
    return AttentionPlan(tiles[0], tiles[1])


class WindowAttention:
    """Weights of one attention mixer. ``w_in``: rows ``[q | k | v | gate]`` of a stacked input projection, every head ``hd``
    wide (the gate has one row per padded head); ``w_o`` [width, heads_pad * hd]."""

    def __init__(self, cfg: WindowAttentionConfig, tensors: dict, hd: int, width_pad: int, device, dtype):
        c = self.cfg = cfg
        self.hd = hd
        G, Gp, KH = c.heads // c.kv_heads, c.group_pad, c.kv_heads

        def rows(t, group, group_pad, d):                  # [KH * group * d, width] -> padded heads
            t = t.view(KH, group, d, t.shape[1])
            return F.pad(t, (0, width_pad - t.shape[3], 0, hd - d, 0, group_pad - group)).reshape(-1, width_pad)

        per_head = lambda t: F.pad(t.view(KH, G), (0, Gp - G)).reshape(-1)
        parts = [rows(tensors["q"], G, Gp, c.dim), rows(tensors["k"], 1, 1, c.dim), rows(tensors["v"], 1, 1, c.vdim)]
        self.g_off = (c.heads_pad + 2 * KH) * hd
        if c.head_gate:
            g = F.pad(tensors["g"].view(KH, G, -1), (0, width_pad - tensors["g"].shape[1], 0, Gp - G)).reshape(-1, width_pad)
            parts.append(F.pad(g, (0, 0, 0, up8(c.heads_pad) - c.heads_pad)))
        self.w_in = torch.cat(parts)
        o = tensors["o"]
        o = F.pad(o.view(o.shape[0], KH, G, c.vdim), (0, hd - c.vdim, 0, Gp - G)).reshape(o.shape[0], -1)
        self.w_o = F.pad(o, (0, 0, 0, width_pad - o.shape[0])).to(device=device, dtype=dtype).contiguous()
        self.k_off, self.v_off = c.heads_pad * hd, (c.heads_pad + KH) * hd
        self.in_rows = self.w_in.shape[0]
        self.sink = torch.zeros(c.heads_pad, dtype=torch.float32, device=device) if c.zero_sink else None
        if c.sink:
            self.sink = per_head(tensors["sink"].float()).to(device=device).contiguous()
        self.bias = None
        if c.bias:
            column = lambda n, *a: rows(tensors[n + ".b"].float().view(-1, 1), *a)[:, 0]
            parts = [column("q", G, Gp, c.dim), column("k", 1, 1, c.dim), column("v", 1, 1, c.vdim)]
            self.bias = torch.cat(parts).to(device=device, dtype=torch.float32).contiguous()
        norm = lambda t: F.pad(t, (0, hd - c.dim)).to(device=device, dtype=dtype).contiguous()
        self.q_norm, self.k_norm = (norm(tensors["q.norm"]), norm(tensors["k.norm"])) if c.qk_norm else (None, None)

    def prep(self, px, positions, cos_sin, slots, kv, plane: int):
        """Norms and rotation of the queries in place, and of the keys on their way into the cache with the values."""
        c = self.cfg
        block_prep(px, c.heads_pad, self.k_off, self.v_off, c.kv_heads, c.rot_dims, positions, cos_sin, slots, kv, plane,
                   q_norm=self.q_norm, k_norm=self.k_norm, norm_dim=c.dim, eps=c.eps, halves=c.halves,
                   bias=self.bias)

    def __call__(self, q, kv, plane: int, block_table, q_start, q_len, kv_len, plan: Optional[AttentionPlan], out=None, gate=None):
        """q [T, heads_pad * hd]: rotated queries; the step's keys and values are in the cache. Returns [T, heads_pad * hd]."""
        c = self.cfg
        if out is None:
            out = torch.empty(q.shape[0], self.w_o.shape[1], dtype=q.dtype, device=q.device)
        return window_attention(q, kv, plane, block_table, q_start, q_len, kv_len, c.heads_pad, c.kv_heads, c.scale, c.window,
                                self.sink, plan, out, gate, c.out_mult)


def window_attention(q, kv, plane, block_table, q_start, q_len, kv_len, heads, kv_heads, scale, window=0, sink=None, plan=None, out=None,
                     gate=None, gate_mult=1.0):
    hd = kv.shape[5]
    if out is None:
        out = torch.empty(q.shape[0], heads * hd, dtype=q.dtype, device=q.device)
    if q.is_cuda:
        p = plan or AttentionPlan()
        _lib().window_attention(q, out, kv, plane, block_table, q_start, q_len, kv_len, p.tile_seq, p.tile_q0, p.decode_seq, heads,
                                kv_heads, scale, window, sink, gate, gate_mult)
        return out
    page = kv.shape[4]
    for s in range(q_len.numel()):
        t0, n, total = int(q_start[s]), int(q_len[s]), int(kv_len[s])
        pages = block_table[s, : -(-total // page)].long()
        k, v = (kv[pages, i, plane, :kv_heads].transpose(1, 2).reshape(-1, kv_heads, hd)[:total].float() for i in (0, 1))
        k, v = (t.repeat_interleave(heads // kv_heads, 1) for t in (k, v))
        score = torch.einsum("thd,jhd->htj", q[t0: t0 + n].float().view(n, heads, hd), k) * scale
        dist = torch.arange(total - n, total).view(n, 1) - torch.arange(total).view(1, total)
        score = score.masked_fill((dist < 0) | (dist >= (window or total)), float("-inf"))
        if sink is not None:
            score = torch.cat([score, sink.view(-1, 1, 1).expand(-1, n, 1)], 2)
        w = torch.softmax(score, -1)[..., :total]
        o = torch.einsum("htj,jhd->thd", w, v)
        if gate is not None:
            o = o * (gate_mult * torch.sigmoid(gate[t0: t0 + n].float())).unsqueeze(2)
        out[t0: t0 + n] = o.reshape(n, -1).to(out.dtype)
    return out


def block_prep(x, heads, k_off, v_off, kv_heads, dims, positions, cos_sin, slots, kv, plane, silu=(0, 0), relu2=(0, 0), q_norm=None,
               k_norm=None, norm_dim=0, eps=1e-6, halves=False, bias=None):
    """What lies between the stacked input projection ``x`` of a parallel block and its branches, in one launch: queries
    (columns from 0) rotate in place, keys rotate and go into the cache with the values, ``silu`` and ``relu2`` (squared
    relu) name column ranges (first, count) that are activated in place. ``q_norm`` / ``k_norm`` [head width]: heads are RMS-normed
    over their first ``norm_dim`` columns first. ``halves``: pairs lie ``dims / 2`` apart. These two exclude the activations.
    ``bias`` (fp32, one value per column, with ``halves``) is added to q, k and v first."""
    if x.is_cuda:
        _lib().block_prep(x, 0, heads, k_off, v_off, kv_heads, dims, positions, cos_sin, slots, kv, plane, *silu, *relu2, q_norm=q_norm,
                          k_norm=k_norm, norm_dim=norm_dim, eps=eps, halves=halves, bias=bias)
        return
    T, hd, page = x.shape[0], kv.shape[5], kv.shape[4]
    take = lambda off, n: x[:, off: off + n * hd].float().add(0.0 if bias is None else bias[off: off + n * hd]).reshape(T, n, hd)

    def rotated(t, w):
        t = t.clone()
        if w is not None:
            t *= torch.rsqrt(t.pow(2).sum(-1, keepdim=True) / (norm_dim or hd) + eps) * w.float()
        if dims and halves:
            cs = cos_sin[positions.long()].unsqueeze(1)
            c, s = cs[..., : dims // 2], cs[..., dims // 2:]
            u, v = t[..., : dims // 2].clone(), t[..., dims // 2: dims].clone()
            t[..., : dims // 2], t[..., dims // 2: dims] = u * c - v * s, v * c + u * s
        elif dims:
            cs = cos_sin[positions.long()].unsqueeze(1)
            c, s = cs[..., : dims // 2], cs[..., dims // 2:]
            u, v = t[..., 0:dims:2].clone(), t[..., 1:dims:2].clone()
            t[..., 0:dims:2], t[..., 1:dims:2] = u * c - v * s, v * c + u * s
        return t

    x[:, : heads * hd] = rotated(take(0, heads), q_norm).reshape(T, -1).to(x.dtype)
    k = rotated(take(k_off, kv_heads), k_norm).to(kv.dtype)
    v = take(v_off, kv_heads).to(kv.dtype)
    ok = slots >= 0
    pg, off = slots[ok] // page, slots[ok] % page
    kv[pg, 0, plane, :kv_heads, off] = k[ok]
    kv[pg, 1, plane, :kv_heads, off] = v[ok]
    a, n = silu
    x[:, a: a + n] = F.silu(x[:, a: a + n].float()).to(x.dtype)
    a, n = relu2
    x[:, a: a + n] = torch.relu(x[:, a: a + n].float()).square().to(x.dtype)
