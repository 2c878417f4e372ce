"""Mixture-of-experts layer: routing, expert GEMMs, weighted combine.

``MoE.forward`` runs
    router logits -> top-k (group-limited sigmoid routing for DeepSeek-V3, softmax top-k otherwise)
    -> sort (token, slot) pairs by expert -> gather rows in expert order
    -> grouped gate/up GEMM with SwiGLU epilogue -> grouped down GEMM
    -> un-permute + router-weighted sum (+ shared experts).
On CUDA every stage is one of this package's kernels (``moe.cu`` and the grouped mode of the
tcgen05 GEMM); on CPU the same stages run in PyTorch. ``e_begin`` / ``e_end`` restrict the layer
to the experts this rank owns (expert parallelism): pairs routed elsewhere contribute nothing
locally and are handled by the dispatch / combine exchange in :mod:`modular_b200.parallel.ep`.

Reference: max/python/max/nn/moe/moe.py:221 (``MoE``, forward :743-865), ``MoEGate`` :118,
architectures/deepseekV3/layers/moe_gate.py:36 (group-limited router).
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from .. import ops
from .._native import lib as _lib


@dataclass
class MoEConfig:
    hidden_size: int
    moe_intermediate_size: int
    n_routed_experts: int
    num_experts_per_tok: int
    n_shared_experts: int = 0
    n_group: int = 1
    topk_group: int = 1
    norm_topk_prob: bool = True
    routed_scaling_factor: float = 1.0
    scoring_func: str = "sigmoid"       # sigmoid (DeepSeek-V3) | softmax


# ---------------------------------------------------------------------- reference routing
def route_group_limited_ref(logits, bias, cfg: MoEConfig):
    scores = torch.sigmoid(logits.float())
    choice = scores + (bias.float() if bias is not None else 0.0)
    T, E = scores.shape
    g = choice.view(T, cfg.n_group, E // cfg.n_group)
    gscore = g.topk(min(2, g.shape[-1]), dim=-1).values.sum(-1)
    gidx = gscore.topk(cfg.topk_group, dim=-1).indices
    gmask = torch.zeros_like(gscore, dtype=torch.bool).scatter_(1, gidx, True)
    masked = choice.masked_fill(~gmask.unsqueeze(-1).expand_as(g).reshape(T, E), float("-inf"))
    ids = masked.topk(cfg.num_experts_per_tok, dim=-1).indices
    w = scores.gather(1, ids)
    if cfg.norm_topk_prob:
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    return ids.int(), w * cfg.routed_scaling_factor


def route_softmax_ref(logits, cfg: MoEConfig):
    p = torch.softmax(logits.float(), dim=-1)
    w, ids = p.topk(cfg.num_experts_per_tok, dim=-1)
    if cfg.norm_topk_prob:
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    return ids.int(), w * cfg.routed_scaling_factor


def route_softmax_group_limited(logits, cfg: MoEConfig):
    """DeepSeek-V2's ``group_limited_greedy``: softmax over all experts, the ``topk_group`` groups with the largest
    single score stay, top-k among their experts (torch ops on either device: this router has no kernel of its own)."""
    p = torch.softmax(logits.float(), dim=-1)
    T, E = p.shape
    g = p.view(T, cfg.n_group, E // cfg.n_group)
    gidx = g.amax(dim=-1).topk(cfg.topk_group, dim=-1).indices
    gmask = torch.zeros(T, cfg.n_group, dtype=torch.bool, device=p.device).scatter_(1, gidx, True)
    masked = p.masked_fill(~gmask.unsqueeze(-1).expand_as(g).reshape(T, E), 0.0)
    w, ids = masked.topk(cfg.num_experts_per_tok, dim=-1)
    if cfg.norm_topk_prob:
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    return ids.int(), (w * cfg.routed_scaling_factor).contiguous()


def route(logits, bias, cfg: MoEConfig):
    """Returns (topk_ids int32 [T, k], topk_weights fp32 [T, k])."""
    if cfg.scoring_func != "sigmoid" and cfg.n_group > 1:
        return route_softmax_group_limited(logits, cfg)
    if not logits.is_cuda:
        if cfg.scoring_func == "sigmoid":
            return route_group_limited_ref(logits, bias, cfg)
        return route_softmax_ref(logits, cfg)
    T, k = logits.shape[0], cfg.num_experts_per_tok
    ids = torch.empty(T, k, dtype=torch.int32, device=logits.device)
    w = torch.empty(T, k, dtype=torch.float32, device=logits.device)
    lg = logits.float().contiguous()
    if cfg.scoring_func == "sigmoid":
        _lib().moe_router_group_limited(lg, bias.float() if bias is not None else None, ids, w, cfg.n_group,
                                        cfg.topk_group, cfg.norm_topk_prob, cfg.routed_scaling_factor)
    else:
        _lib().moe_router_softmax_topk(lg, ids, w, cfg.norm_topk_prob)
        if cfg.routed_scaling_factor != 1.0:
            w *= cfg.routed_scaling_factor
    return ids, w


class Fp8ExpertWeights:
    """Block-scaled fp8 weights of a stack of experts: ``q`` [E, N, K] float8_e4m3fn and ``scale`` fp32
    [E, N/128, ceil(K/128)] (the checkpoint's ``weight_scale_inv`` per 128x128 block); N % 128 == 0.
    Reference: max/python/max/nn/moe/moe_fp8.py:48 with the fp8-blockwise strategy of quant_strategy.py."""

    def __init__(self, q: torch.Tensor, scale: torch.Tensor):
        self.q, self.scale = q.contiguous(), scale.float().contiguous()

    @classmethod
    def quantize(cls, w: torch.Tensor) -> "Fp8ExpertWeights":
        qs = [ops.reference.quant_fp8_weight_block128(w[e]) for e in range(w.shape[0])]
        return cls(torch.stack([q for q, _ in qs]), torch.stack([s for _, s in qs]))

    @property
    def shape(self):
        return self.q.shape

    def __getitem__(self, e):
        """Integer: dequantised weight of expert ``e`` (reference paths). Slice: that range of experts."""
        if isinstance(e, slice):
            return Fp8ExpertWeights(self.q[e], self.scale[e])
        return ops.reference.dequant_fp8_weight_block128(self.q[e], self.scale[e])

    def contiguous(self):
        return self


class MoE:
    """Weights: ``gate`` [E, H] router, ``w_gate_up`` [E_local, 2I, H], ``w_down`` [E_local, H, I] (bf16
    tensors or :class:`Fp8ExpertWeights`), optional shared experts fused as one MLP (``shared_gate_up``
    [2 I_s, H], ``shared_down`` [H, I_s])."""

    def __init__(self, cfg: MoEConfig, gate, w_gate_up, w_down, e_score_bias=None, shared_gate_up=None,
                 shared_down=None, e_begin: int = 0, e_end: Optional[int] = None):
        self.cfg = cfg
        self.gate, self.bias = gate, e_score_bias
        self.w_gate_up, self.w_down = w_gate_up, w_down
        self.shared_gate_up, self.shared_down = shared_gate_up, shared_down
        self.e_begin = e_begin
        self.e_end = cfg.n_routed_experts if e_end is None else e_end
        self._scratch = None

    @classmethod
    def random_init(cls, cfg: MoEConfig, device="cpu", dtype=torch.bfloat16, seed=0, std=0.02, **kw):
        g = torch.Generator().manual_seed(seed)
        r = lambda *s: (torch.randn(*s, generator=g) * std).to(dtype).to(device)
        E, H, I = cfg.n_routed_experts, cfg.hidden_size, cfg.moe_intermediate_size
        e0, e1 = kw.get("e_begin", 0), kw.get("e_end") or E
        full_gu, full_d = r(E, 2 * I, H), r(E, H, I)
        shared = cfg.n_shared_experts * I
        return cls(cfg, r(E, H).float().to(device), full_gu[e0:e1].contiguous(), full_d[e0:e1].contiguous(),
                   (torch.randn(E, generator=g) * 0.1).to(device) if cfg.scoring_func == "sigmoid" else None,
                   r(2 * shared, H) if shared else None, r(H, shared) if shared else None, **kw)

    # ------------------------------------------------------------ pieces
    def router_logits(self, x):
        """fp32 router scores [T, E]. On the GPU the product runs on this package's GEMM with a bf16 copy of the
        router matrix (checkpoints store it in bf16, so nothing is lost) and fp32 accumulation and output."""
        if x.is_cuda and x.dtype == torch.bfloat16 and self.gate.shape[0] % 64 == 0:
            if getattr(self, "_gate_bf16", None) is None:
                self._gate_bf16 = self.gate.to(torch.bfloat16).contiguous()
            return ops.linear(x, self._gate_bf16, out_dtype=torch.float32)
        return x.float() @ self.gate.float().t()

    def shared_forward(self, x):
        if self.shared_gate_up is None:
            return None
        if x.is_cuda and x.dtype == torch.bfloat16 and x.shape[0] <= ops.DECODE_GEMM_MAX_TOKENS:
            return ops.linear_decode(ops.linear_decode(x, self.shared_gate_up, "swiglu"), self.shared_down)
        return ops.linear(ops.linear_swiglu(x, self.shared_gate_up), self.shared_down)

    def experts_forward(self, x, ids, w, shared_out=None):
        """Local experts on tokens x with routing (ids, w); returns y [T, H]."""
        if not x.is_cuda:
            return self._experts_ref(x, ids, w, shared_out)
        cfg, dev = self.cfg, x.device
        T, k = ids.shape
        E = self.e_end - self.e_begin
        if self._scratch is None or self._scratch[0].device != dev:
            self._scratch = (torch.zeros(2 * E, dtype=torch.int32, device=dev),
                             torch.empty(E + 1, dtype=torch.int32, device=dev))
        scratch, offsets = self._scratch
        order = torch.empty(T * k, dtype=torch.int32, device=dev)
        inverse = torch.empty(T * k, dtype=torch.int32, device=dev)
        L = _lib()
        L.moe_create_indices(ids, self.e_begin, self.e_end, scratch, offsets, order, inverse)
        n_local = offsets[E:E + 1]
        xp = torch.empty(T * k, cfg.hidden_size, dtype=x.dtype, device=dev)
        L.moe_permute_rows(x, order, n_local, xp, k)
        out = self.local_gemms(xp, offsets)
        y = torch.empty(T, cfg.hidden_size, dtype=x.dtype, device=dev)
        L.moe_combine(out, inverse, w, shared_out, y, k)
        return y

    def local_gemms(self, xp, offsets, act=None, out=None, max_rows: int = 0, expected_rows: int = 0):
        """Both grouped GEMMs of the local experts on rows already in expert order (``offsets`` int32
        [E_local + 1]). ``xp``: bf16 rows, or ``(xq, xs)`` = e4m3 rows [n, H] (any row stride) with fp32
        scales [H/128, n] for fp8 experts that receive quantised rows. Returns bf16 [n, H]. ``n`` may be an
        upper bound of the rows (the true count is ``offsets[-1]`` on the device); ``max_rows`` bounds the rows
        of one expert and ``expected_rows`` is the typical count per expert (it picks the token tile)."""
        cfg, L = self.cfg, _lib()
        fp8_in = isinstance(xp, tuple)
        n = (xp[0] if fp8_in else xp).shape[0]
        dev = (xp[0] if fp8_in else xp).device
        if out is None:
            out = torch.empty(n, cfg.hidden_size, dtype=torch.bfloat16, device=dev)
        if isinstance(self.w_gate_up, Fp8ExpertWeights):
            # quantise per 1x128 group, grouped block-scaled GEMM, SwiGLU, quantise again, second grouped
            # GEMM (rows past the local count hold garbage that is never read back)
            xq, xs = xp if fp8_in else ops.quant_fp8_group128(xp)
            I = cfg.moe_intermediate_size
            E = self.e_end - self.e_begin
            bn = 0
            if expected_rows > 0:
                bn = 32 if expected_rows <= 32 else (64 if expected_rows <= 64 else 128)
            gu = torch.empty(n, 2 * I, dtype=torch.bfloat16, device=dev)
            L.grouped_gemm_fp8(xq, xs, self.w_gate_up.q, self.w_gate_up.scale, gu, offsets, max_rows or n, bn)
            # SwiGLU and the quantisation of its result in one pass over the rows that exist
            aq = torch.empty(n, I, dtype=torch.float8_e4m3fn, device=dev)
            a_s = torch.empty(I // 128, n, dtype=torch.float32, device=dev)
            L.silu_mul_quant_fp8(gu, aq, a_s, offsets[E:E + 1])
            L.grouped_gemm_fp8(aq, a_s, self.w_down.q, self.w_down.scale, out, offsets, max_rows or n, bn)
            return out
        if fp8_in:
            raise ValueError("quantised rows need fp8 expert weights")
        if act is None:
            act = torch.empty(n, cfg.moe_intermediate_size, dtype=xp.dtype, device=dev)
        L.grouped_gemm_bf16(xp, self.w_gate_up, act, offsets, n, True, 0)
        L.grouped_gemm_bf16(act, self.w_down, out, offsets, n, False, 0)
        return out

    def _experts_ref(self, x, ids, w, shared_out=None):
        cfg = self.cfg
        y = torch.zeros(x.shape[0], cfg.hidden_size, dtype=torch.float32, device=x.device)
        if shared_out is not None:
            y += shared_out.float()
        I = cfg.moe_intermediate_size
        for e in range(self.e_begin, self.e_end):
            tok, slot = torch.nonzero(ids == e, as_tuple=True)
            if tok.numel() == 0:
                continue
            xe = x[tok]
            gu = self.w_gate_up[e - self.e_begin]
            h = ops.reference.linear_swiglu(xe, gu)
            o = ops.reference.linear(h, self.w_down[e - self.e_begin])
            y.index_add_(0, tok, o.float() * w[tok, slot].unsqueeze(1))
        return y.to(x.dtype)

    def forward(self, x):
        ids, w = route(self.router_logits(x), self.bias, self.cfg)
        return self.experts_forward(x, ids, w, self.shared_forward(x))

    __call__ = forward


# ---------------------------------------------------------------------- routing by token id
class TableRouter:
    """Experts chosen by a table of token ids (no scores: the ``top`` experts of an id weigh ``1 / top`` each) for all the
    mixture-of-experts layers of a model. Since the choice does not depend on activations, one kernel sorts the pairs of
    every layer before the first layer runs, and the layers' norm and residual kernels read and write expert order
    directly. ``tables``: one int tensor [vocab, top] and the expert count per layer."""

    def __init__(self, tables: list, experts: list, device):
        dev = torch.device(device)
        self.experts = list(experts)
        self.tops = [int(t.shape[1]) for t in tables]
        self.tables = [t.to(dev, torch.int32).contiguous() for t in tables]
        self._flat = torch.cat([t.reshape(-1) for t in self.tables]) if tables else None
        desc, first, pairs, offs = [], 0, 0, 0
        for t, e in zip(self.tables, self.experts):
            desc.append([first, t.shape[1], e, pairs, offs, t.shape[0]])
            first, pairs, offs = first + t.numel(), pairs + t.shape[1], offs + e + 1
        self._desc = torch.tensor(desc, dtype=torch.int64, device=dev).view(-1, 6)
        self._pairs, self._offs = pairs, offs

    def route(self, ids: torch.Tensor) -> list:
        """Per layer: (inverse int32 [T, top]: row of every pair in expert order, offsets int32 [experts + 1])."""
        if not self.tables:
            return []
        T = ids.numel()
        if not ids.is_cuda:
            return [self._route_ref(ids, t, e) for t, e in zip(self.tables, self.experts)]
        inverse = torch.empty(T * self._pairs, dtype=torch.int32, device=ids.device)
        offsets = torch.empty(self._offs, dtype=torch.int32, device=ids.device)
        _lib().moe_table_route(ids, self._flat, self._desc, max(self.experts), inverse, offsets)
        out, p, o = [], 0, 0
        for top, e in zip(self.tops, self.experts):
            out.append((inverse[T * p: T * (p + top)].view(T, top), offsets[o: o + e + 1]))
            p, o = p + top, o + e + 1
        return out

    @staticmethod
    def _route_ref(ids, table, experts):
        flat = table[ids.long()].reshape(-1).long()
        order = torch.argsort(flat, stable=True)
        inverse = torch.empty_like(order)
        inverse[order] = torch.arange(order.numel())
        offsets = torch.zeros(experts + 1, dtype=torch.int32)
        offsets[1:] = torch.cumsum(torch.bincount(flat, minlength=experts), 0)
        return inverse.view(-1, table.shape[1]).int(), offsets


@dataclass
class ScoreRouterConfig:
    """Sigmoid scores (``softmax``: a softmax over all candidates), a choice among the ``keep`` best of ``groups`` groups of
    neighbouring candidates (a group counts its two best choice scores, or with ``group_max`` its best one), weights from the scores
    without the correction. The candidates are the experts and, behind them, ``identity`` identity experts, which give the input back
    and have no weights."""
    experts: int
    top: int
    groups: int = 1
    keep: int = 1
    renormalize: bool = False
    scaling: float = 1.0
    softmax: bool = False
    group_max: bool = False
    identity: int = 0

    def __post_init__(self):
        n = self.candidates
        if self.experts < 1 or self.identity < 0 or self.groups < 1 or n % self.groups:
            raise ValueError(f"{n} experts cannot form {self.groups} equal groups")
        if not 1 <= self.keep <= self.groups or not 1 <= self.top <= self.keep * (n // self.groups):
            raise ValueError(f"{self.top} experts out of {self.keep} groups of {n // self.groups}")
        if self.top > 32 or n > 1024:
            raise ValueError("at most 32 of at most 1024 experts per token")

    @property
    def candidates(self) -> int:
        return self.experts + self.identity


class ScoreRouter:
    """Router of one layer for experts whose rows are kept in expert order: ``route`` goes from the router's input to the rows
    of every expert; the layer's seam weighs and adds what comes back."""

    def __init__(self, cfg: ScoreRouterConfig, gate, correction, width_pad: int, device, dtype):
        self.cfg = cfg
        E8 = (cfg.candidates + 7) // 8 * 8
        self.gate = F.pad(gate, (0, width_pad - gate.shape[1], 0, E8 - gate.shape[0])).to(device=device, dtype=dtype).contiguous()
        self.correction = None if correction is None else correction.to(device=device, dtype=torch.float32).contiguous()

    def choose_reference(self, logits):
        """logits [T, candidates] -> (candidates chosen [T, top], weights fp32 [T, top])."""
        c, z = self.cfg, logits.float()
        scores = torch.softmax(z, -1) if c.softmax else torch.sigmoid(z)
        choice = scores if self.correction is None else scores + self.correction
        g = choice.view(z.shape[0], c.groups, -1)
        best = g.topk(1 if c.group_max else min(2, g.shape[2]), dim=-1).values.sum(-1)
        kept = torch.zeros_like(best, dtype=torch.bool).scatter_(1, best.topk(c.keep, dim=-1).indices, True)
        ids = g.masked_fill(~kept.unsqueeze(-1), float("-inf")).reshape(z.shape).topk(c.top, dim=-1).indices
        w = scores.gather(1, ids)
        if c.renormalize:
            w = w / (w.sum(-1, keepdim=True) + 1e-20)
        return ids, w * c.scaling

    def route(self, x, counts):
        """x [T, width]; ``counts`` int32 [experts], zero. Returns (rows [T * top, width] in expert order, offsets int32
        [experts + 1], inverse int32 [T, top]: row of every pair (-1: an identity expert), weights fp32 [T, top])."""
        c, T, dev = self.cfg, x.shape[0], x.device
        logits = ops.linear(x, self.gate, out_dtype=torch.float32)
        if not x.is_cuda:
            ids, w = self.choose_reference(logits[:, : c.candidates])
            flat = ids.reshape(-1)
            order = torch.argsort(flat, stable=True)             # identity experts come last
            inverse = torch.empty_like(order)
            inverse[order] = torch.arange(order.numel())
            inverse[flat >= c.experts] = -1
            offsets = torch.zeros(c.experts + 1, dtype=torch.int32)
            offsets[1:] = torch.cumsum(torch.bincount(flat, minlength=c.candidates)[: c.experts], 0)
            return x[order // c.top], offsets, inverse.view(T, c.top).int(), w
        i32 = lambda *s: torch.empty(*s, dtype=torch.int32, device=dev)
        ids, rank, inverse, offsets = i32(T, c.top), i32(T, c.top), i32(T, c.top), i32(c.experts + 1)
        w = torch.empty(T, c.top, dtype=torch.float32, device=dev)
        L = _lib()
        L.moe_score_route(logits, self.correction, ids, w, rank, counts, c.groups, c.keep, c.renormalize, c.scaling, c.softmax,
                          c.group_max, c.identity)
        rows = torch.empty(T * c.top, x.shape[1], dtype=x.dtype, device=dev)
        L.moe_place_rows(x, ids, rank, counts, offsets, inverse, rows)
        return rows, offsets, inverse, w


def expert_mlp(xp, offsets, w_gate_up, w_down, max_rows: int):
    """SwiGLU experts on rows already in expert order: xp [rows, H] -> [rows, H]; w_gate_up [E, 2I, H], w_down [E, H, I].
    ``max_rows`` bounds the rows of one expert (the step's tokens when a token's experts differ)."""
    n, I = xp.shape[0], w_gate_up.shape[1] // 2
    out = torch.empty(n, w_down.shape[1], dtype=xp.dtype, device=xp.device)
    if not xp.is_cuda:
        out.zero_()
        off = offsets.tolist()
        for e in range(w_down.shape[0]):
            if off[e + 1] > off[e]:
                out[off[e]: off[e + 1]] = ops.reference.linear(
                    ops.reference.linear_swiglu(xp[off[e]: off[e + 1]], w_gate_up[e]), w_down[e])
        return out
    act = torch.empty(n, I, dtype=xp.dtype, device=xp.device)
    L = _lib()
    if xp.dtype == torch.float32:
        gu = torch.empty(n, 2 * I, dtype=xp.dtype, device=xp.device)
        L.grouped_gemm_f32(xp, w_gate_up, gu, offsets)
        L.silu_mul_f32(gu, act)
        L.grouped_gemm_f32(act, w_down, out, offsets)
    else:
        L.grouped_gemm_bf16(xp, w_gate_up, act, offsets, max_rows, True, 0)
        L.grouped_gemm_bf16(act, w_down, out, offsets, max_rows, False, 0)
    return out


def gated_mlp(x, w_gate_up, w_down):
    """One SwiGLU feed-forward: x [T, H], w_gate_up [2I, H], w_down [H, I]."""
    if x.is_cuda and x.dtype == torch.float32:
        return ops.linear(ops.silu_mul(ops.linear(x, w_gate_up)), w_down)
    return ops.linear(ops.linear_swiglu(x, w_gate_up), w_down)
