"""Mavidra against the plain implementation in ``mavidra_oracle``: every mechanism alone, then whole models through the engine's
own step (portions, mixed batches, reused pages and slots, window edges, long decoding) and greedy generation through its
scheduler. CPU runs take the package's PyTorch operations in fp32; GPU runs take the kernels in fp32 and bf16."""

import copy
import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import mavidra_oracle as oracle  # noqa: E402
from modular_b200 import ops
from modular_b200.entrypoints.llm import LLM
from modular_b200.entrypoints.trace import TraceSession
from modular_b200.kv_cache import KVCacheParams, PagedKVCacheManager
from modular_b200.models.mavidra import MavidraConfig, MavidraWeights
from modular_b200.nn.bigram import BigramConfig, bigram_rows
from modular_b200.nn.delta_rule import DeltaRule, DeltaRuleConfig
from modular_b200.nn.gated_linear_attention import GatedLinearAttention, GatedLinearConfig
from modular_b200.nn.latent_attention import LatentAttention, latent_attention
from modular_b200.nn.moe import ScoreRouter, ScoreRouterConfig, expert_mlp
from modular_b200.nn.parallel_mixer import ParallelMixer
from modular_b200.nn.residual import sandwich_norm
from modular_b200.nn.rotary_embedding import cos_sin_table
from modular_b200.nn.window_attention import WindowAttention, block_prep, tensor_core_plan, window_attention
from modular_b200.pipelines.context import SamplingParams, TextContext
from modular_b200.pipelines.registry import PIPELINE_REGISTRY
from modular_b200.pipelines.weights import save_checkpoint

RUNS = [pytest.param("cpu", torch.float32, id="cpu-fp32"),
        pytest.param("cuda:0", torch.float32, id="gpu-fp32", marks=pytest.mark.gpu),
        pytest.param("cuda:0", torch.bfloat16, id="gpu-bf16", marks=pytest.mark.gpu)]
TOL = {torch.float32: 2e-4, torch.bfloat16: 3e-2}        # root mean square error over that of the expected values


def rel(got, want):
    got, want = got.double().cpu(), want.double()
    return ((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp(min=1e-12)).item()


def i32(*v):
    return torch.tensor(v, dtype=torch.int32)


def rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def double(t):
    return {k: v.double() for k, v in t.items()}


# ---------------------------------------------------------------------------------- configurations and weights
def moe(experts=6, top=2, groups=3, keep=2, ff=72):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}


def gla(heads=3, dim=20, vdim=28, tau=12.0):
    return {"type": "gla", "mixer": dict(heads=heads, dim=dim, vdim=vdim, tau=tau)}


def latent(heads=3, dim=40, rot_dim=24, vdim=20, kv_rank=72, q_rank=56, window=37, base=900.0, scale=None, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale or (dim + rot_dim) ** -0.5,
             mask={"size": window}, rot={"base": base, "dims": rot_dim})
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def parallel(heads=6, kv_heads=2, dim=40, vdim=24, dims=16, base=3000.0, scale=None, rheads=4, rkv=2, rdim=20, rvdim=28, conv=4, ls=0.7, rs=1.3):
    left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5, rot={"base": base, "dims": dims})
    right = dict(heads=rheads, kv_heads=rkv, dim=rdim, vdim=rvdim, conv=conv)
    return {"type": "parallel", "mixer": dict(left=left, right=right, left_scale=ls, right_scale=rs)}


def config(*layers, width=104, vocab=190, eps=1e-5, mult=0.6, scale=0.7, bigram=(83, 29, 5)):
    """Layers are mixers (followed by the usual experts) or pairs (mixer, feed-forward or None)."""
    out = []
    for l in layers:
        m, ff = l if isinstance(l, tuple) else (l, moe())
        out.append({**copy.deepcopy(m), "mlp": copy.deepcopy(ff)})
    return {"architecture": "Mavidra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"scale": scale, "bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "layers": out}


def weights_for(cfg, seed=0, rank=20, dtype=torch.bfloat16):
    """Random tensors of a checkpoint, rounded to ``dtype``; scores, decays and logits such that a wrong key or state shows."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    c, t = MavidraConfig.from_hf(cfg), {}
    for name, shape in c.tensor_shapes({i: rank for i in c.of_type("gla")}).items():
        leaf = name.split(".", 2)[-1] if name.startswith("l") else name
        if name.endswith("a2.b"):
            v = rnd(*shape)
        elif leaf.endswith(".b") and len(shape) == 1 or leaf in ("norm1.b", "norm2.b", "norm1b.b", "norm2b.b"):
            v = 0.3 * rnd(*shape)
        elif leaf.endswith("A_log"):
            v = 0.5 * rnd(*shape) - 1.0
        elif leaf.endswith("dt_bias"):
            v = rnd(*shape) - 2.0
        elif leaf.endswith("correction"):
            v = 0.3 * rnd(*shape) - 0.4                              # choice scores on both sides of zero
        elif leaf.endswith("sink"):
            v = 1.0 + rnd(*shape)
        elif "norm" in leaf:
            v = 1.0 + 0.2 * rnd(*shape)
        elif leaf.endswith(".conv"):
            v = rnd(*shape) * shape[-1] ** -0.5
        elif name in ("embed", "bigram"):
            v = rnd(*shape)
        else:
            v = rnd(*shape) * shape[-1] ** -0.5
            if leaf.endswith(("uq", "left.q", "router")):
                v = 2.0 * v
        t[name] = v
    return {k: v.to(dtype).float() for k, v in t.items()}


def part(t, prefix):
    return {k[len(prefix):]: v for k, v in t.items() if k.startswith(prefix)}


def paged(n_tokens, page, seed=0):
    """A block table of shuffled pages for one sequence: (table [1, n], pages in the pool, slots of every position)."""
    n = -(-n_tokens // page)
    pages = torch.randperm(n + 2, generator=torch.Generator().manual_seed(seed))[:n].int()
    pos = torch.arange(n_tokens)
    return pages.view(1, -1), n + 2, pages.long()[pos // page] * page + pos % page


def two_sequences(lens, steps):
    """Walks the steps (lists of (name, tokens)) of two sequences: rows per entry and q_start / q_len / kv_len."""
    at = dict.fromkeys(lens, 0)
    for step in steps:
        rows = [(s, at[s], at[s] + n) for s, n in step]
        for s, n in step:
            at[s] += n
        ql = i32(*[n for _, n in step])
        yield rows, (torch.cumsum(ql, 0) - ql).int(), ql, i32(*[hi for _, _, hi in rows])
    assert at == lens


STEPS = ([("a", 2)], [("a", 1), ("b", 30)], [("b", 2), ("a", 67)], [("a", 1), ("b", 1)], [("b", 7), ("a", 2)], [("a", 1)], [("a", 1)])
STEP_LENS = {"a": 75, "b": 40}


# ---------------------------------------------------------------------------------- embedding and seams
@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda:0", marks=pytest.mark.gpu)])
def test_bigram_rows(device):
    """Two sequences in portions; slots that held another request's last token before; a sequence without a slot."""
    c = BigramConfig(1009, 1 << 20, 77)
    toks = {"a": torch.randint(0, 1 << 30, (75,), generator=torch.Generator().manual_seed(0)), "b": torch.arange(40)}
    spec = dict(buckets=1009, mul_prev=1 << 20, mul_cur=77)
    want = {s: oracle.bigram_rows(v.tolist(), spec) for s, v in toks.items()}
    last, slot, got = torch.full((5, 1), 12345, device=device), {"a": 3, "b": 0}, {"a": [], "b": []}
    for rows, qs, ql, kl in two_sequences(STEP_LENS, STEPS):
        x = torch.cat([toks[s][lo:hi] for s, lo, hi in rows]).to(device)
        idx = i32(*[slot[s] for s, _, _ in rows]).to(device)
        out = bigram_rows(c, x, qs.to(device), ql.to(device), kl.to(device), idx, last).tolist()
        for (s, lo, hi), o in zip(rows, qs.tolist()):
            got[s] += out[o: o + hi - lo]
    assert got == want and want["a"][0] == want["b"][0] == 1009 and max(want["a"][1:]) < 1009
    assert last.flatten().tolist() == [39, 12345, 12345, int(toks["a"][-1]), 12345]
    one = lambda *v: i32(*v).to(device)
    assert bigram_rows(c, torch.tensor([7], device=device), one(0), one(1), one(5), one(-1), last).tolist() == [1009]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("width,center", [(64, True), (203, True), (200, False), (1336, True), (5000, True), (4100, False)])
def test_sandwich_seam(width, center, device, dtype):
    """Embedding with rows of a second table, a normed branch, weighted experts in expert order, some rows only."""
    T, V, pad, eps, k = 7, 20, (width + 7) // 8 * 8, 1e-3, 3
    r = lambda i, *s: torch.nn.functional.pad(rand(*s, width, seed=width + i), (0, pad - width)).to(dtype)
    table, second, a, e = r(0, V), r(1, 9), 0.02 * r(2, T) + 0.05 * r(9, 1), r(3, T * k)      # a: mean not zero, eps matters
    wu, bu, w1, b1 = r(4, 1)[0], r(5, 1)[0], r(6, 1)[0], r(7, 1)[0]
    norm = ((lambda x, w, b: oracle.layer_norm(x, w, b, eps)) if center else (lambda x, w, b: oracle.rms(x, w, eps)))
    ids = torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(0))
    ids2 = torch.tensor([8, 0, 3, 8, 1, 1, 5])
    inverse = torch.randperm(T * k, generator=torch.Generator().manual_seed(1)).view(T, k).int()
    pw = torch.rand(T, k, generator=torch.Generator().manual_seed(2))
    D, d = (lambda t: t.to(device)), (lambda t: t[..., :width].double())
    B = lambda b: D(b) if center else None
    x, n1 = torch.empty(T, pad, device=device), torch.empty(T, pad, dtype=dtype, device=device)
    kw = dict(cols=width, eps=eps)
    sandwich_norm(x, ids=D(ids), table=D(table), scale=0.3, inject_ids=D(ids2), inject=D(second), w1=D(w1), b1=B(b1), n1=n1, **kw)
    h = 0.3 * d(table)[ids] + d(second)[ids2]
    assert rel(x[:, :width], h) < 1e-6 and rel(n1[:, :width], norm(h, d(w1), d(b1))) < TOL[dtype]
    sandwich_norm(x, a=D(a), w_u=D(wu), b_u=B(bu), mult=0.4, w1=D(w1), b1=B(b1), n1=n1, **kw)
    h = h + 0.4 * norm(d(a), d(wu), d(bu))
    assert rel(x[:, :width], h) < 2e-6 and rel(n1[:, :width], norm(h, d(w1), d(b1))) < TOL[dtype]
    u = (d(e)[inverse.long()] * pw.double().unsqueeze(2)).sum(1)
    y = x.clone()
    sandwich_norm(y, e=D(e), inverse=D(inverse), pair_w=D(pw), w_u=D(wu), b_u=B(bu), mult=0.4, **kw)
    h = h + 0.4 * norm(u, d(wu), d(bu))
    assert rel(y[:, :width], h) < 2e-6
    rows, out, before = i32(6, 0, 6), torch.empty(3, pad, dtype=dtype, device=device), x.clone()
    sandwich_norm(x, e=D(e), inverse=D(inverse), pair_w=D(pw), w_u=D(wu), b_u=B(bu), mult=0.4, rows=D(rows), w1=D(w1), b1=B(b1), n1=out,
                  store_x=False, **kw)
    assert torch.equal(x, before) and rel(out[:, :width], norm(h, d(w1), d(b1))[[6, 0, 6]]) < TOL[dtype]
    assert (out[:, width:] == 0).all() and (y[:, width:] == 0).all()
    sandwich_norm(x, a=D(a), mult=0.5, **kw)                                               # a branch without a norm of its own
    assert rel(x[:, :width], before[:, :width].double().cpu() + 0.5 * d(a)) < 1e-6


# ---------------------------------------------------------------------------------- softmax attention
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("hd,dim,dims,halves", [(64, 40, 16, True), (64, 64, 64, True), (128, 100, 6, True), (128, 72, 0, True), (64, 48, 24, False),
                                                (168, 168, 50, True)])
def test_normed_and_rotated_heads(hd, dim, dims, halves, device, dtype):
    """Per-head norms over the true width before the rotation, values untouched, the store into shuffled pages."""
    T, H, KH, page, first, eps = 9, 5, 2, 64, 300, 1e-2
    cs = cos_sin_table(dims, first + T, 500.0, None, device) if dims else None
    x = torch.zeros(T, H + 2 * KH, hd)
    x[..., :dim] = 0.2 * rand(T, H + 2 * KH, dim, seed=dims)
    x = x.to(dtype)
    wq, wk = (torch.nn.functional.pad(1.0 + 0.3 * rand(dim, seed=s), (0, hd - dim)).to(dtype) for s in (1, 2))
    y, x = x.reshape(T, -1).clone().to(device), x.double()
    kv = torch.full((8, 2, 3, KH, page, hd), 5.0, dtype=dtype, device=device)
    slots = torch.randperm(8 * page, generator=torch.Generator().manual_seed(1))[:T]
    slots[4] = -1
    block_prep(y, H, H * hd, (H + KH) * hd, KH, dims, torch.arange(first, first + T, dtype=torch.int32, device=device), cs, slots.to(device),
               kv, 1, q_norm=wq.to(device), k_norm=wk.to(device), norm_dim=dim, eps=eps, halves=halves)
    turn = lambda t, w: oracle.rotate(oracle.rms(t[..., :dim], w[:dim].double(), eps), dict(dims=dims, base=500.0), first, halves)
    assert rel(y.view(T, -1, hd)[:, :H, :dim], turn(x[:, :H], wq)) < TOL[dtype] and (y.view(T, -1, hd)[:, :H, dim:] == 0).all()
    k, v, c = turn(x[:, H: H + KH], wk), x[:, H + KH:], kv.cpu().double()
    for t in range(T):
        if t != 4:
            pg, o = int(slots[t]) // page, int(slots[t]) % page
            assert rel(c[pg, 0, 1, :, o, :dim], k[t]) < TOL[dtype] and rel(c[pg, 1, 1, :, o], v[t]) == 0
    assert int((c != 5.0).any(-1).sum()) == 2 * KH * (T - 1) and (c[:, :, [0, 2]] == 5.0).all()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,KH,hd", [(4, 2, 64), (16, 1, 64), (8, 4, 128), (3, 3, 160), (16, 2, 128)])
@pytest.mark.parametrize("sink", [-40.0, 2.0, 60.0])
def test_gate_and_sink_of_softmax_attention(H, KH, hd, sink, device, dtype):
    """Gate and sink per head where prompts and decoded tokens go through different kernels; a far key stands out."""
    T, page = 200, 64
    bt, pages, slots = paged(T, page, seed=3)
    q, k, v = (0.3 * rand(T, n, hd, seed=n + i).to(dtype).double() for i, n in enumerate((H, KH, KH)))
    k[5] = q[150, :KH] = q[199, :KH] = 1.0                       # a score of hd / 8 for a key far back
    sinks, gate = sink + torch.arange(H).float(), rand(T, H, seed=9).to(dtype)
    kv = torch.zeros(pages * page, 2, KH, hd, dtype=torch.float64)
    kv[slots, 0], kv[slots, 1] = k, v
    kv = kv.view(pages, page, 2, KH, hd).permute(0, 2, 3, 1, 4).unsqueeze(2).contiguous().to(device, dtype)
    want = oracle.grouped_attention(q, k, v, 0.125, sinks.double()) * 0.7 * oracle.sigmoid(gate.double()).unsqueeze(2)
    D, at = (lambda *x: i32(*x).to(device)), 0
    for n in (130, 2, 66, 1, 1):
        plan = tensor_core_plan(H // KH, hd, dtype, page, D(0), D(n), n, n == 1)
        got = window_attention(q[at: at + n].reshape(n, -1).to(device, dtype), kv, 0, bt.to(device), D(0), D(n), D(at + n), H, KH, 0.125, 0,
                               sinks.to(device), plan, gate=gate[at: at + n].to(device), gate_mult=0.7)
        exp = want[at: at + n].reshape(n, -1)
        if exp.abs().max() > 1e-12:
            assert rel(got, exp) < TOL[dtype]
        else:
            assert got.abs().max() < 1e-10
        at += n


def run_parallel(cfg, device, dtype, pieces, T, seed=1):
    W, page = cfg["width"], 64
    t, c = weights_for(cfg, seed=seed), MavidraConfig.from_hf(cfg)
    a, d, hd = c.attention(0), c.delta(0), c.head_width
    mix = ParallelMixer(WindowAttention(a, part(t, "l0.mix.left."), hd, W, device, dtype), DeltaRule(d, part(t, "l0.mix.right."), W, device, dtype),
                        device, dtype)
    h = rand(T, W, seed=2).to(dtype)
    want = oracle.parallel_mixer(h.double(), double(t), "l0.mix.", cfg["layers"][0]["mixer"], cfg["norm"]["eps"])
    bt, pages, slots = paged(T, page)
    kv = torch.zeros(pages, 2, 1, a.kv_heads, page, hd, dtype=dtype, device=device)
    state, conv = (torch.ones((1, *d.state_shapes()[n]), device=device) for n in ("delta", "conv"))
    cs = cos_sin_table(a.rot_dims, T, a.rope_base, None, device)
    D, got, at = (lambda *v: i32(*v).to(device)), [], 0
    for n in pieces:
        plan = tensor_core_plan(a.group_pad, hd, dtype, page, D(0), D(n), n, n == 1)
        got.append(mix(h[at: at + n].to(device), ops.linear, kv, 0, state, conv, cs, torch.arange(at, at + n, dtype=torch.int32, device=device),
                       slots[at: at + n].to(device), bt.to(device), D(0), D(n), D(at + n), D(0), plan, n == 1)[:, :W])
        at += n
    return torch.cat(got), want


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("m", [parallel(), parallel(heads=1, kv_heads=1, dim=8, vdim=8, dims=2, rheads=1, rkv=1, rdim=8, rvdim=8, conv=1),
                               parallel(heads=5, kv_heads=1, dim=72, vdim=128, dims=72, rheads=6, rkv=2, rdim=128, rvdim=72, conv=2, ls=-0.5, rs=0.3),
                               parallel(heads=6, kv_heads=3, dim=160, vdim=40, dims=100, rheads=3, rkv=1, rdim=33, rvdim=17, conv=5),
                               parallel(heads=34, kv_heads=2, dim=16, vdim=32, dims=8, rheads=40, rkv=8, rdim=24, rvdim=8, ls=1.0, rs=1.0)],
                         ids=["odd", "small", "wide", "wide head", "many heads"])
def test_parallel_mixer(m, device, dtype):
    got, want = run_parallel(config(m), device, dtype, (85, 2, 61, 1, 1), 150)
    assert rel(got, want) < TOL[dtype]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,KH,d,dv,taps", [(4, 4, 32, 32, 4), (6, 2, 24, 40, 3), (3, 1, 72, 9, 2), (2, 2, 128, 128, 4), (2, 1, 100, 136, 1),
                                            (1, 1, 300, 16, 5), (36, 12, 64, 64, 3), (2, 2, 200, 264, 4)])
def test_delta_rule_with_a_decay_per_head(H, KH, d, dv, taps, device, dtype):
    """Two sequences in portions beside each other, in slots that held something else before."""
    W = 104
    cfg = config(parallel(rheads=H, rkv=KH, rdim=d, rvdim=dv, conv=taps), width=W)
    t, c = weights_for(cfg, seed=H), DeltaRuleConfig(W, H, KH, d, dv, taps, 0, 0, 1e-5, head_decay=True, out_mult=0.8)
    mix, w = DeltaRule(c, part(t, "l0.mix.right."), W, device, dtype), double(t)
    h = {s: rand(n, W, seed=n).to(dtype) for s, n in STEP_LENS.items()}
    want = {s: 0.8 * oracle.right_mixer(x.double(), w, "l0.mix.right.", cfg["layers"][0]["mixer"]["right"], 1e-5) for s, x in h.items()}
    state, conv = (torch.full((5, *c.state_shapes()[n]), 3.0, device=device) for n in ("delta", "conv"))
    slot, got = {"a": 3, "b": 1}, {"a": [], "b": []}
    for rows, qs, ql, kl in two_sequences(STEP_LENS, STEPS):
        x = torch.cat([h[s][lo:hi] for s, lo, hi in rows]).to(device)
        y = mix(x, ops.linear, state, conv, i32(*[slot[s] for s, _, _ in rows]).to(device), qs.to(device), ql.to(device), kl.to(device),
                bool((ql == 1).all()))
        for (s, lo, hi), o in zip(rows, qs.tolist()):
            got[s].append(y[o: o + hi - lo, :W])
    for s in h:
        assert rel(torch.cat(got[s]), want[s]) < TOL[dtype], s
    assert (state[[0, 2, 4]] == 3.0).all() and (conv[[0, 2, 4]] == 3.0).all()       # nobody else's slot was written


# ---------------------------------------------------------------------------------- gated linear attention
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,d,dv,tau,rank", [(3, 20, 28, 12.0, 20), (1, 8, 8, 1.0, 1), (5, 32, 64, 16.0, 16), (2, 128, 128, 4.0, 72), (4, 48, 9, 0.5, 8),
                                             (2, 100, 136, 30.0, 40), (1, 300, 16, 16.0, 16), (2, 200, 264, 2.0, 16)])
def test_gated_linear_mixer(H, d, dv, tau, rank, device, dtype):
    """Two sequences in portions beside each other, in slots that held something else before; slow and very fast decays."""
    W = 104
    cfg = config(gla(H, d, dv, tau), width=W)
    t, c = weights_for(cfg, seed=d, rank=rank), GatedLinearConfig(H, d, dv, rank, tau, 1e-5)
    t["l0.mix.a2.b"] += torch.linspace(-30.0, 6.0, H * d)[torch.randperm(H * d, generator=torch.Generator().manual_seed(1))]
    mix, w = GatedLinearAttention(c, part(t, "l0.mix."), W, device, dtype), double(t)
    lens, steps = {"a": 275, "b": 140}, ([("a", 2)], [("a", 1), ("b", 130)], [("b", 2), ("a", 267)], [("a", 1), ("b", 1)], [("b", 7), ("a", 2)],
                                         [("a", 1)], [("a", 1)])
    h = {s: rand(n, W, seed=n).to(dtype) for s, n in lens.items()}
    want = {s: oracle.gla_mixer(x.double(), w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5) for s, x in h.items()}
    state = torch.full((5, *c.state_shapes()["gla"]), 3.0, device=device)
    slot, got = {"a": 3, "b": 1}, {"a": [], "b": []}
    for rows, qs, ql, kl in two_sequences(lens, steps):
        x = torch.cat([h[s][lo:hi] for s, lo, hi in rows]).to(device)
        y = mix(x, ops.linear, state, i32(*[slot[s] for s, _, _ in rows]).to(device), qs.to(device), ql.to(device), kl.to(device),
                bool((ql == 1).all()))
        for (s, lo, hi), o in zip(rows, qs.tolist()):
            got[s].append(y[o: o + hi - lo, :W])
    for s in h:
        assert rel(torch.cat(got[s]), want[s]) < TOL[dtype], s
    assert (state[[0, 2, 4]] == 3.0).all()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("gap", [1, 15, 16, 63, 64, 65, 130, 300])
def test_gated_linear_attention_remembers_one_token(gap, device, dtype):
    """One key and value far back and a query that asks for it: what is left after ``gap`` decays, in prompts and decoding."""
    H, d, dv, T = 2, 32, 16, 340
    c = GatedLinearConfig(H, d, dv, 4, 16.0, 1e-5)
    g = torch.Generator().manual_seed(gap)
    q, k, v = (0.02 * torch.randn(T, H, n, generator=g) for n in (d, d, dv))
    z = 4.0 + torch.randn(T, H * d, generator=g)
    k[20], v[20], q[20 + gap] = 1.0, torch.randn(H, dv, generator=g), 1.0
    q, k, v = (x.to(dtype) for x in (q, k, v))
    alpha = torch.exp(-oracle.softplus(-z.double()) / 16.0).view(T, H, d)
    want, S = oracle.gla_scan(q.double() * d ** -0.5, k.double(), v.double(), alpha)
    want = oracle.rms(want, 1.0, 1e-5).reshape(T, -1)
    zero = lambda *s: torch.zeros(*s)
    mix = GatedLinearAttention(c, {"q": zero(H * d, 8), "k": zero(H * d, 8), "v": zero(H * dv, 8), "g": zero(H * dv, 8), "o": zero(8, H * dv),
                                   "norm": torch.ones(dv), "a1": zero(4, 8), "a2": zero(H * d, 4), "a2.b": zero(H * d)}, 64, device, dtype)
    px = torch.zeros(T, mix.a_off + 64, dtype=dtype)
    px[:, : H * d], px[:, mix.k_off: mix.v_off] = q.reshape(T, -1), k.reshape(T, -1)
    px[:, mix.v_off: mix.g_off], px[:, mix.g_off: mix.a_off] = v.reshape(T, -1), 50.0         # silu(50) = 50
    D = lambda *x: i32(*x).to(device)
    for pieces in ((T,), (20 + gap, T - 20 - gap), (21, 1, gap - 1, T - 21 - gap) if gap > 1 else (21, 1, T - 22), (21 + gap, 2, T - 23 - gap)):
        state, got, at = torch.full((1, *c.state_shapes()["gla"]), 9.0, device=device), [], 0
        for n in pieces:
            out = torch.empty(n, H * dv, dtype=dtype, device=device)
            mix.mix(px[at: at + n].to(device), z[at: at + n].to(device), out, state, D(0), D(0), D(n), D(at + n), n == 1)
            got.append(out.double().cpu() / 50.0)
            at += n
        y = torch.cat(got)
        assert rel(y[20 + gap], want[20 + gap]) < TOL[dtype], pieces
        assert rel(y[200:], want[200:]) < 2 * TOL[dtype], pieces
        assert rel(state[0, :, :, :d].transpose(1, 2), S) < 2e-5
    assert rel(oracle.rms(oracle.gla_scan(q[21:].double(), k[21:].double(), v[21:].double(), alpha[21:])[0], 1.0, 1e-5).reshape(T - 21, -1)[gap - 1],
               want[20 + gap]) > 0.2                                                            # without that token: something else


@pytest.mark.gpu
@pytest.mark.parametrize("H,d,dv", [(2, 8, 8), (3, 64, 64), (5, 96, 72), (2, 128, 128), (1, 40, 200), (4, 32, 256)])
@pytest.mark.parametrize("pace", [0.02, 1.0, 6.0, 40.0])
def test_gated_linear_chunks_agree_with_the_scan(H, d, dv, pace):
    """Chunks on the tensor cores against the fp32 token loop on the same values: sequences that begin, go on, end inside a chunk or
    have one token, decays from none to all within a token (some channels fast beside slow ones)."""
    from modular_b200._native import lib

    lens, old, slots = [150, 1, 64, 2, 200, 63], [0, 5, 64, 7, 130, 1], [3, 0, 5, -1, 1, 6]
    T = sum(lens)
    r = lambda *s, seed: rand(*s, seed=seed).cuda()
    cols = H * (2 * d + 2 * dv)
    x, w = r(T, cols, seed=d).bfloat16(), (1.0 + 0.1 * r(dv, seed=1)).bfloat16()
    z = pace * torch.where(torch.arange(H * d).cuda() % 3 > 0, -1.0, 0.3) * r(T, H * d, seed=2).abs()
    bias, pad = r(H * d, seed=3), next(n for n in (32, 64, 96, 128) if d <= n)
    idx, ql = i32(*slots).cuda(), i32(*lens).cuda()
    kl, qs = (ql + i32(*old).cuda()).int(), (torch.cumsum(ql, 0) - ql).int()
    init = r(8, H, dv, pad, seed=4)
    init[..., d:] = 0
    got = []
    for dtype in (torch.bfloat16, torch.float32):
        xx, st = x.to(dtype), init.clone()
        o, out = torch.empty(T, H * dv, device="cuda"), torch.empty(T, H * dv, dtype=dtype, device="cuda")
        lib().gla(xx, 0, H * d, 2 * H * d, z, bias, d ** -0.5, 1.0, xx[:, H * (2 * d + dv):], True, 0.9, w.to(dtype), 1e-5, dv, o, out, st, idx, qs,
                  ql, kl, H, d, dv, False)
        got.append((o, out, st))
    assert rel(got[0][2], got[1][2].cpu()) < 2e-5 and rel(got[0][0], got[1][0].cpu()) < 3e-5 and rel(got[0][1], got[1][1].cpu()) < 5e-3
    assert torch.equal(got[0][2][[2, 4, 7]], init[[2, 4, 7]]) and got[0][2].isfinite().all()


@pytest.mark.parametrize("device,dtype", RUNS)
def test_recurrences_without_a_slot(device, dtype):
    """Sequences with slot -1 start from zero and keep nothing (the dummies of a padded decode batch)."""
    W = 104
    cfg = config(gla(), parallel(), width=W)
    t, D = weights_for(cfg), lambda *v: i32(*v).to(device)
    w, eps = double(t), 1e-5
    c, d = GatedLinearConfig(3, 20, 28, 20, 12.0, eps), MavidraConfig.from_hf(cfg).delta(1)
    one, two = GatedLinearAttention(c, part(t, "l0.mix."), W, device, dtype), DeltaRule(d, part(t, "l1.mix.right."), W, device, dtype)
    state, s2, conv = (torch.ones((2, *s), device=device) for s in (c.state_shapes()["gla"], *d.state_shapes().values()))
    for lens in ((1, 1), (70, 3)):
        x = rand(sum(lens), W).to(device, dtype)
        args = (D(-1, -1), D(0, lens[0]), D(*lens), D(lens[0], 99), lens == (1, 1))
        y, y2 = one(x, ops.linear, state, *args), two(x, ops.linear, s2, conv, *args)
        for lo, hi in ((0, lens[0]), (lens[0], sum(lens))):
            h = x[lo: hi].cpu().double()
            assert rel(y[lo: hi, :W], oracle.gla_mixer(h, w, "l0.mix.", cfg["layers"][0]["mixer"], eps)) < TOL[dtype]
            assert rel(y2[lo: hi, :W], 1.3 * oracle.right_mixer(h, w, "l1.mix.right.", cfg["layers"][1]["mixer"]["right"], eps)) < TOL[dtype]
    assert (state == 1).all() and (s2 == 1).all() and (conv == 1).all()


# ---------------------------------------------------------------------------------- latent attention
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("m", [latent(), latent(heads=1, dim=8, rot_dim=8, vdim=8, kv_rank=16, q_rank=8, window=1),
                               latent(heads=7, dim=130, rot_dim=64, vdim=100, kv_rank=300, q_rank=200, window=64),
                               latent(heads=2, dim=32, rot_dim=72, vdim=32, kv_rank=64, q_rank=96, window=65),
                               latent(heads=16, dim=64, rot_dim=32, vdim=64, kv_rank=520, q_rank=64, window=400)],
                         ids=["odd", "small", "wide", "rot72", "latent520"])
def test_latent_mixer(m, device, dtype):
    """One mixer over a prompt in portions and decoded tokens, and a second one with a window of its own on its cache rows."""
    other = latent(**{**{k: m["mixer"][k] for k in ("rot_dim", "kv_rank", "q_rank")}, "heads": 3, "dim": 24, "vdim": 36, "window": 50, "kv_from": 0})
    cfg = config(m, other)
    t, c, W, T, page = weights_for(cfg, seed=1), MavidraConfig.from_hf(cfg), 104, 150, 64
    mixers = [LatentAttention(c.latent(i), part(t, f"l{i}.mix."), W, device, dtype) for i in (0, 1)]
    h, w = rand(T, W, seed=2).to(dtype), double(t)
    rows = oracle.latent_rows(h.double(), w, "l0.mix.", m["mixer"], 1e-5)
    want = [oracle.latent_mixer(h.double(), w, f"l{i}.mix.", cfg["layers"][i]["mixer"], 1e-5, rows) for i in (0, 1)]
    bt, pages, slots = paged(T, page)
    cache = torch.full((pages, 2, page, c.latent(0).cache_width + 8), 7.0, dtype=dtype, device=device)
    cs = cos_sin_table(m["mixer"]["rot_dim"], T, 900.0, None, device)
    D, got, at = (lambda *v: i32(*v).to(device)), ([], []), 0
    for n in (85, 2, 61, 1, 1):
        for i, mix in enumerate(mixers):
            got[i].append(mix(h[at: at + n].to(device), ops.linear, cache[:, 1], cs, torch.arange(at, at + n, dtype=torch.int32, device=device),
                              slots[at: at + n].to(device), bt.to(device), D(0), D(n), D(at + n), n == 1)[:, :W])
        at += n
    for i in (0, 1):
        assert rel(torch.cat(got[i]), want[i]) < TOL[dtype], i
    assert (cache[:, 0] == 7.0).all()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 100, 500])
@pytest.mark.parametrize("heads,rank", [(3, 128), (128, 512), (5, 64)])
def test_one_latent_key_at_the_edge_of_the_window(heads, rank, window, device, dtype):
    """One key stands out for every query: it must be seen up to ``window - 1`` tokens later and not after that, in prompts, from
    portions and from decoding, also where it lies at a page border."""
    page, T = 64, 260
    gen = torch.Generator().manual_seed(window)
    rows, q = 0.05 * torch.randn(T, rank + 64, generator=gen), 0.05 * torch.randn(T, heads, rank + 64, generator=gen)
    mark = torch.zeros(rank + 64)
    mark[3] = mark[rank + 2] = 4.0                                 # half of the score from the latent, half from the rotated part
    bt, pages, slots = paged(T, page, seed=6)
    D = lambda *v: i32(*v).to(device)
    for place in (0, 63, 64, 130):
        r, qq = rows.clone(), (q + mark).to(dtype).float()
        r[place] += mark
        r = r.to(dtype).float()
        cache = torch.zeros(pages * page, rank + 64)
        cache[slots] = r
        cache = cache.view(pages, page, -1).to(device, dtype)
        last = min(place + window - 1, T - 2)                      # the last query that sees it
        starts = sorted({s for s in (last - 1, last, last + 1) if s >= place})
        s = torch.einsum("qhd,kd->hqk", qq, r).double()
        p = oracle.softmax(torch.where(oracle.visible(T, window), s, torch.full_like(s, -1e30)))
        want = torch.einsum("hqk,kd->qhd", p, r[:, :rank].double())
        assert want[last, :, 3].min() > 3.0 and (last + 1 > place + window - 1) == (want[last + 1, :, 3].max() < 1.0)
        spans = [(0, T)] + [(a, a + n) for a in starts for n in (1, 2) if a + n <= T] + [(max(last - 70, 0), last + 2)]
        for lo, hi in spans:
            x = qq[lo: hi].to(device, dtype)
            got = latent_attention(x[..., :rank].contiguous(), x[..., rank:].contiguous(), cache, bt.to(device), D(0), D(hi - lo), D(hi), 1.0,
                                   None, hi - lo == 1, window)
            err = (got.double().cpu() - want[lo: hi]).abs().amax((1, 2))
            assert err.max() < (1e-4 if dtype == torch.float32 else 6e-2), (place, lo, hi, lo + int(err.argmax()))


@pytest.mark.gpu
@pytest.mark.parametrize("heads,rank", [(128, 512), (12, 512), (6, 192), (96, 384), (67, 64)])
@pytest.mark.parametrize("decode", [True, False])
@pytest.mark.parametrize("window", [0, 1, 64, 200])
def test_latent_attention_kernels_agree(heads, rank, decode, window):
    """The tensor-core kernels (split over the keys or not) against the CUDA-core kernel on the same rows, with windows and gates."""
    g = torch.Generator(device="cuda").manual_seed(9)
    lens, qn = [700, 1, 64, 65, 333], [1] * 5 if decode else [150, 1, 64, 2, 100]
    page, need = 64, [-(-n // 64) for n in lens]
    bt = torch.zeros(5, max(need), dtype=torch.int32, device="cuda")
    perm = torch.randperm(sum(need), generator=torch.Generator().manual_seed(1)).int().cuda()
    for b, n in enumerate(need):
        bt[b, :n] = perm[sum(need[:b]): sum(need[:b]) + n]
    rows = lambda *s: torch.randn(*s, generator=g, device="cuda", dtype=torch.float32).bfloat16()
    cache, T = rows(sum(need), page, rank + 64), sum(qn)
    q, gate, sink = rows(T, heads, rank + 64), rows(T, heads), torch.randn(heads, generator=g, device="cuda")
    ql, kl = torch.tensor(qn, dtype=torch.int32, device="cuda"), torch.tensor(lens, dtype=torch.int32, device="cuda")
    qs = (torch.cumsum(ql, 0) - ql).int()
    for sk in (None, sink):
        args = (bt, qs, ql, kl, (rank + 64) ** -0.5, sk, decode, window)
        got = latent_attention(q[..., :rank].contiguous(), q[..., rank:].contiguous(), cache, *args, gate)
        want = latent_attention(q[..., :rank].float().contiguous(), q[..., rank:].float(), cache.float(), *args, gate.float())
        assert rel(got, want.cpu()) < 1e-2


# ---------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("experts,top,groups,keep,ff", [(6, 2, 3, 2, 72), (8, 4, 2, 1, 24), (1, 1, 1, 1, 64), (40, 7, 5, 2, 16), (64, 8, 1, 1, 8),
                                                        (96, 3, 96, 40, 8), (260, 10, 4, 2, 8), (16, 16, 4, 4, 8)])
def test_grouped_router_and_experts(experts, top, groups, keep, ff, device, dtype):
    """The choice (choice scores on both sides of zero), the weights, the order of the rows, and the weighted sum."""
    W, T = 96, 77
    cfg = config((gla(), moe(experts, top, groups, keep, ff)), width=W)
    t = weights_for(cfg, seed=2)
    t["l0.mlp.router"] *= 4.0
    r, w = cfg["layers"][0]["mlp"]["router"], double(t)
    x = rand(T, W, seed=1).to(dtype)
    router = ScoreRouter(ScoreRouterConfig(experts, top, groups, keep), t["l0.mlp.router"], t["l0.mlp.correction"], W, device, dtype)
    rows, offsets, inverse, weights = router.route(x.to(device), torch.zeros(experts, dtype=torch.int32, device=device))
    inv, off, weights = inverse.cpu().long(), offsets.cpu().tolist(), weights.cpu()
    assert sorted(inv.flatten().tolist()) == list(range(T * top)) and off[0] == 0 and off[-1] == T * top
    assert torch.equal(rows.cpu()[inv], x.unsqueeze(1).expand(T, top, W))
    s = oracle.sigmoid(x.double() @ w["l0.mlp.router"].T)
    clear = 0
    for i in range(T):
        if oracle.choice_margin(s[i], w["l0.mlp.correction"], r) < 1e-4:
            continue
        clear += 1
        mine = [next(e for e in range(experts) if off[e] <= p < off[e + 1]) for p in inv[i].tolist()]
        assert sorted(mine) == sorted(oracle.choose(s[i], w["l0.mlp.correction"], r))
        assert torch.allclose(weights[i].double(), s[i, mine], rtol=1e-4, atol=1e-6)
    assert clear > T // 2
    gu = torch.stack([torch.cat([t[f"l0.mlp.e{e}.gate"], t[f"l0.mlp.e{e}.up"]]) for e in range(experts)])
    dn = torch.stack([t[f"l0.mlp.e{e}.down"] for e in range(experts)])
    pad = max(64, ff) - ff
    gu = torch.nn.functional.pad(gu.view(experts, 2, ff, W), (0, 0, 0, pad)).reshape(experts, -1, W)
    out = expert_mlp(rows, offsets, gu.to(device, dtype), torch.nn.functional.pad(dn, (0, pad)).to(device, dtype), T).cpu().double()
    got = (out[inv] * weights.double().unsqueeze(2)).sum(1)
    want = oracle.moe(x.double(), w, "l0.mlp.", cfg["layers"][0]["mlp"])
    err = (got - want).pow(2).mean(1).sqrt() / want.pow(2).mean().sqrt()
    assert err.sort().values[: int(0.9 * T)].max() < TOL[dtype]


def test_router_config_checks():
    for bad in (dict(experts=6, top=2, groups=4, keep=1), dict(experts=6, top=3, groups=3, keep=1), dict(experts=6, top=2, groups=3, keep=4),
                dict(experts=6, top=0), dict(experts=64, top=33), dict(experts=2048, top=2)):
        with pytest.raises(ValueError):
            ScoreRouterConfig(**bad)


# ---------------------------------------------------------------------------------- whole models
MIXED = config(gla(), latent(), parallel(), (latent(heads=4, dim=24, vdim=56, window=64, q_rank=40, kv_from=1), None),
               (parallel(heads=4, kv_heads=4, dim=24, vdim=56, dims=24, rheads=2, rkv=1, rdim=40, rvdim=16, conv=2, ls=1.1, rs=0.4), moe(8, 3, 2, 1, 40)),
               (latent(heads=2, dim=16, rot_dim=16, vdim=48, kv_rank=136, q_rank=72, window=3, base=70.0), moe(5, 1, 1, 1)),
               latent(heads=3, dim=32, vdim=16, window=100, kv_from=1, base=900.0), (gla(2, 72, 40, 4.0), moe(4, 4, 2, 2, 88)))


def clear_choices(t, dtype):
    """Runs that round would choose other experts where two choices are close, and such a token changes all that follow: their
    experts depend on the corrections (the choice itself has a test of its own, and fp32 runs choose by token)."""
    return t if dtype == torch.float32 else {k: (20.0 * v).bfloat16().float() if k.endswith("correction") else v for k, v in t.items()}


@functools.cache
def mixed_reference(dtype):
    t = clear_choices(weights_for(MIXED), dtype)
    draw = lambda n, s: torch.randint(0, MIXED["vocab"], (n,), generator=torch.Generator().manual_seed(s)).tolist()
    out = {}
    for r, toks in (("a", draw(300, 3)), ("b", draw(150, 4))):
        out[r] = (toks, *oracle.forward(MIXED, t, toks), functools.cache(lambda toks=toks: rounding_noise(MIXED, t, toks)))
    return t, out


@pytest.fixture(scope="module")
def mixed_model():
    return mixed_reference


def engine(cfg, t, device, dtype, tokens=512, page=64, batch=4, **kw):
    c = MavidraConfig.from_hf(cfg)
    args = dict(max_length=tokens, max_batch_size=batch, max_batch_input_tokens=tokens, page_size=page,
                num_kv_pages=-(-tokens // page) + 1, enable_prefix_caching=False, max_logit_rows=tokens,
                enable_overlap_scheduler=False, graph_batch_sizes=[1, 4])
    args.update(kw)
    return LLM(c, MavidraWeights.from_state_dict(c, t, device, dtype), device=device, dtype=dtype, **args)


def rounding_noise(cfg, t, tokens, samples=3):
    """How far rounding the operands and results of matrix products to 16 bits moves the rows of the plain implementation:
    (logits, stream), the largest of some samples. Recurrences normed over a few tokens, and close choices of experts, move a lot."""
    exact, out = oracle.forward(cfg, t, tokens), None
    for i in range(samples):
        g = torch.Generator().manual_seed(i)
        oracle.ROUND = lambda x: x * (1.0 + 2.0 ** -8 * (torch.rand(x.shape, generator=g, dtype=x.dtype) - 0.5))
        try:
            got = oracle.forward(cfg, t, tokens)
        finally:
            oracle.ROUND = lambda x: x
        err = [(a - b).pow(2).mean(-1).sqrt() for a, b in zip(got, exact)]
        out = err if out is None else [torch.maximum(a, b) for a, b in zip(out, err)]
    return out


def check_rows(got, want, noise, dtype, what=""):
    """Every row in fp32; in bf16 nearly every row within what rounding does to it."""
    err, unit = (got.double().cpu() - want).pow(2).mean(-1).sqrt(), want.pow(2).mean().sqrt()
    if dtype == torch.float32:
        assert err.max() < 5e-4 * unit, (what, int(err.argmax()))
        return
    ratio = err / torch.maximum(4.0 * noise(), TOL[dtype] * unit)
    assert (ratio < 1.0).double().mean() > 0.95 and err.median() < 2.0 * torch.maximum(noise().median(), 0.01 * unit), (what, ratio, err / unit)


def replay(llm, reqs, steps):
    """Runs ``steps`` (lists of (request, tokens)) and returns every request's logits [T, vocab]; all places are wanted. A
    request ends with its last token, so its pages and slot are free for the next one."""
    s, at, out = TraceSession(llm), {}, {}
    for step in steps:
        entries, end = [], []
        for r, n in step:
            toks, lo = reqs[r.split("#")[0]], at.get(r, 0)
            entries.append({"id": r, "tokens": toks[lo: lo + n], "want": list(range(n))})
            at[r] = lo + n
            if at[r] == len(toks):
                end.append(r)
        logits, row = s.step(entries, end).cpu(), 0
        for r, n in step:
            out.setdefault(r, []).append(logits[row: row + n])
            row += n
    assert not s.live and llm.kv.used_blocks_pct == 0 and llm.kv.free_state_slots == 4
    return {r: torch.cat(v) for r, v in out.items()}


@pytest.mark.parametrize("device,dtype", RUNS)
def test_residual_stream_of_every_layer(mixed_model, device, dtype):
    t, ref = mixed_model(dtype)
    toks, _, want, noise = ref["b"]
    llm = engine(MIXED, t, device, dtype)
    ctx = TextContext.from_prompt(toks, llm.max_length, "r")
    llm.kv.claim(ctx)
    llm.kv.alloc(ctx)
    b = llm.pipeline.packer.step_tensors(llm.pipeline.packer.pack([ctx], llm.kv))
    stream = []
    llm.model._forward(b["tokens"], b["positions"], b["slots"], b["block_table"], b["q_start"], b["q_len"], b["kv_len"],
                       b["logit_rows"], b["state_slot"], stream=stream)
    assert len(stream) == len(want) == 8 and stream[0].dtype == torch.float32
    for i, (got, exp) in enumerate(zip(stream, want)):
        check_rows(got, exp, lambda: noise()[1][i], dtype, f"after layer {i}")


def cut(n, *sizes):
    """Portions of the given sizes, repeated, that add up to n."""
    out, i = [], 0
    while n:
        k = min(n, sizes[i % len(sizes)])
        out.append(k)
        n, i = n - k, i + 1
    return out


SCHEDULES = {
    "whole": [[("a", 300)], [("b", 150)]],
    "token by token": [[("b", 1)]] * 150,
    "long decoding": [[("a", 20)]] + [[("a", 1)]] * 280,
    "twos": [[("a", n)] for n in cut(300, 2)],
    "page borders": [[("a", n)] for n in cut(300, 63, 1, 1, 63, 2, 62, 64)],
    "changing": [[("a", n)] for n in cut(300, 2, 3, 50, 2, 17, 5)],
    "mixed": [[("a", 100), ("b", 3)], [("b", 60), ("a", 1)], [("a", 1), ("b", 1)], [("b", 2), ("a", 90)], [("a", 1)], [("b", 84), ("a", 107)]],
    "reuse": [[("a", 200), ("b", 70)], [("b", 80), ("a", 2)], [("b#2", 2), ("a", 40)], [("a", 1), ("b#2", 1)], [("a", 57), ("b#2", 40)],
              [("b#2", 107), ("b#3", 9)], [("a#2", 150), ("b#3", 1)], [("a#2", 1), ("b#3", 1)], [("b#3", 139)], [("a#2", 149)]],
}


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", SCHEDULES)
def test_schedules(mixed_model, name, device, dtype):
    t, ref = mixed_model(dtype)
    out = replay(engine(MIXED, t, device, dtype), {r: v[0] for r, v in ref.items()}, SCHEDULES[name])
    for r, got in out.items():
        _, want, _, noise = ref[r.split("#")[0]]
        check_rows(got, want, lambda: noise()[0], dtype, r)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("cfg", [
    config(gla()), config(latent()), config(parallel()),
    config((parallel(heads=1, kv_heads=1, dim=4, vdim=4, dims=2, rheads=1, rkv=1, rdim=4, rvdim=4, conv=1), moe(1, 1, 1, 1, 4)),
           (gla(1, 4, 4, 1.0), None), (latent(1, 4, 2, 4, 4, 4, 1), moe(2, 1, 2, 1, 4)), width=42, vocab=33, bigram=(1, 0, 0)),
    config(latent(), (latent(heads=6, dim=100, vdim=8, kv_from=0, window=70), None), latent(kv_rank=200, rot_dim=64, window=2), eps=1e-3, width=136, vocab=258,
           mult=1.0, scale=2.0),
    config((parallel(heads=10, kv_heads=2, dim=104, vdim=80, dims=60, rheads=7, rkv=7, rdim=104, rvdim=48), moe(12, 5, 4, 3, 136)), gla(7, 104, 48, 9.0),
           width=202, vocab=98, bigram=(500, 499, 3)),
    config(parallel(dim=200, vdim=144, dims=66, rheads=2, rdim=144, rvdim=8), parallel(heads=3, kv_heads=1, dim=32, vdim=32, dims=32), width=88)],
    ids=["gla only", "latent only", "parallel only", "tiny", "latent", "wide", "wide heads"])
def test_other_sizes(cfg, device, dtype):
    t = clear_choices(weights_for(cfg, seed=11, rank=9), dtype)
    toks = torch.randint(0, cfg["vocab"], (170,), generator=torch.Generator().manual_seed(1)).tolist()
    want = oracle.forward(cfg, t, toks)[0]
    out = replay(engine(cfg, t, device, dtype), {"a": toks}, [[("a", n)] for n in (40, 2, 1, 1, 21, 1, 104)])
    check_rows(out["a"], want, lambda: rounding_noise(cfg, t, toks)[0], dtype)


@pytest.mark.parametrize("device,dtype", [RUNS[0], RUNS[2]])
def test_pages_of_other_sizes(device, dtype):
    """Pages that are a multiple of 64 tokens and pages that are not (no tensor-core softmax attention then)."""
    cfg = config(latent(window=50), parallel(), gla())
    t = clear_choices(weights_for(cfg, seed=12), dtype)
    toks = torch.randint(0, cfg["vocab"], (260,), generator=torch.Generator().manual_seed(1)).tolist()
    want = oracle.forward(cfg, t, toks)[0]
    for page in (128, 40):
        out = replay(engine(cfg, t, device, dtype, page=page), {"a": toks}, [[("a", n)] for n in (129, 1, 1, 60, 69)])
        check_rows(out["a"], want, lambda: rounding_noise(cfg, t, toks)[0], dtype, page)


def mistakes():
    """Configurations and weights of one planted mistake each."""
    def window(c, t):
        c["layers"][1]["mixer"]["mask"]["size"] += 1

    def sink(c, t):
        t["l2.mix.left.sink"] -= 100.0

    def bigram(c, t):
        c["embedding"]["bigram"]["mul_prev"] = 0

    def side(c, t):
        c["layers"][2]["mixer"]["right_scale"] = 0.0

    def shared(c, t):
        c["layers"][3]["mixer"]["mask"]["size"] -= 1

    def tau(c, t):
        c["layers"][0]["mixer"]["tau"] *= 1.2

    def groups(c, t):
        c["layers"][0]["mlp"]["router"]["groups"]["keep"] = 3

    def bias(c, t):
        t["l4.norm1b.b"] *= 0.0

    def correction(c, t):
        t["l1.mlp.correction"] *= 0.0

    return [window, sink, bigram, side, shared, tau, groups, bias, correction]


@pytest.mark.parametrize("plant", mistakes(), ids=lambda f: f.__name__)
def test_the_comparison_notices_mistakes(mixed_model, plant):
    """A mistake planted in the plain implementation is larger than what the whole-model tests accept."""
    t, ref = mixed_model(torch.float32)
    toks, want = ref["b"][:2]
    c, w = copy.deepcopy(MIXED), {k: v.clone() for k, v in t.items()}
    plant(c, w)
    got = oracle.forward(c, w, toks)[0]
    err = (got - want).pow(2).mean(1).sqrt() / want.pow(2).mean().sqrt()
    assert err.max() > 20 * 5e-4 and (err > 5e-4).double().mean() > 0.2


@pytest.mark.parametrize("device,dtype", RUNS)
def test_greedy_generation(device, dtype):
    """More requests than a batch holds through the scheduler, prompts in chunks beside decoding, with preemption when the
    pool runs dry: the tokens are those of plain greedy decoding."""
    cfg = config(gla(), latent(window=30), (parallel(), None), (latent(heads=2, kv_from=1), None), vocab=150)
    t = clear_choices(weights_for(cfg, seed=21), dtype)
    g = torch.Generator().manual_seed(8)
    prompts = [torch.randint(0, 150, (n,), generator=g).tolist() for n in (70, 1, 50, 60, 5, 90)]
    # 3 state slots and 3 sequences at a time; the 4 pages are full when the third request needs its second one
    llm = engine(cfg, t, device, dtype, tokens=128, batch=3, max_batch_input_tokens=40, enable_in_flight_batching=True,
                 graph_batch_sizes=[2, 3], num_kv_pages=5, max_logit_rows=0)
    recs = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=24, ignore_eos=True))
    exact = total = 0
    for p, r in zip(prompts, recs):
        assert len(r.tokens) == 24
        want = oracle.forward(cfg, t, p + r.tokens)[0][len(p) - 1: -1]
        top, chosen = want.max(-1).values, want[torch.arange(24), r.tokens]
        if dtype == torch.float32:
            assert (top - chosen).max() < 1e-3                                            # never worse than a near tie
        exact += int((want.argmax(-1) == torch.tensor(r.tokens)).sum())
        total += 24
    assert exact >= total * (1.0 if dtype == torch.float32 else 0.85)
    assert llm.kv.free_state_slots == 3 and llm.kv.used_blocks_pct == 0 and llm.kv.preemptions > 0
    if device != "cpu":
        assert llm.model.graph_replays > 0


@pytest.mark.gpu
def test_sampling_and_penalties_on_gpu():
    cfg = config(gla(), latent(), parallel())
    llm = engine(cfg, weights_for(cfg), "cuda:0", torch.bfloat16, max_logit_rows=0)
    sp = lambda seed: SamplingParams(temperature=1.0, top_k=20, max_new_tokens=16, ignore_eos=True, seed=seed, repetition_penalty=1.2)
    a, b = (llm.generate([[1, 2, 3], [4, 5]], [sp(s), sp(s + 1)]) for s in (5, 9))
    assert all(len(r.tokens) == 16 and 0 <= min(r.tokens) and max(r.tokens) < cfg["vocab"] for r in a + b)
    assert [r.tokens for r in a] != [r.tokens for r in b]


# ---------------------------------------------------------------------------------- cache, configuration, command line
def test_paged_tensors_of_the_cache():
    p = KVCacheParams(2, 3, 8, 16, torch.float32, False, False, paged_specs=(("rows", 5, 24),))
    assert p.bytes_per_page == (2 * 2 * 3 * 8 + 5 * 24) * 16 * 4
    kv = PagedKVCacheManager(p, 7)
    assert kv.paged["rows"].shape == (7, 5, 16, 24) and kv.kv.shape == (7, 2, 2, 3, 16, 8)
    with pytest.raises(ValueError):
        PagedKVCacheManager(KVCacheParams(2, 3, 8, 16, torch.float32, False, True, paged_specs=(("rows", 5, 24),)), 7, host_pages=2)


def test_config_checks_and_registry():
    arch = PIPELINE_REGISTRY.retrieve_architecture(MIXED)
    assert arch.name == "Mavidra" and arch.config_class is MavidraConfig
    c = MavidraConfig.from_hf(MIXED)
    again = MavidraConfig.from_hf(c.to_hf())
    assert again.layers == c.layers and again.bigram == c.bigram and PIPELINE_REGISTRY.retrieve_architecture(c.to_hf()) is arch
    assert c.latent_layers == (1, 5) and c.of_type("parallel") == (2, 4) and c.head_width == 64 and c.cache_heads == 4
    assert c.paged_specs() == (("latent", 2, 192 + 64),) and [s[0] for s in c.state_specs()] == [
        "last_token", "l0.gla", "l2.delta", "l2.conv", "l4.delta", "l4.conv", "l7.gla"]
    t = weights_for(MIXED)
    for bad in (config(parallel(heads=5, kv_heads=2)), config(parallel(rheads=3, rkv=2)), config(parallel(dims=50)), config(latent(kv_from=0)),
                config(latent(), latent(kv_from=0, kv_rank=64)), config(latent(), latent(kv_from=0), latent(kv_from=1)),
                config((gla(), moe(6, 5, 3, 2))), config((gla(), moe(6, 2, 4, 2)))):
        with pytest.raises(ValueError):
            MavidraConfig.from_hf(bad)
    with pytest.raises(KeyError):
        MavidraWeights.from_state_dict(c, {k: v for k, v in t.items() if k != "l2.mix.right.norm"}, "cpu", torch.float32)
    with pytest.raises(ValueError):
        MavidraWeights.from_state_dict(c, {**t, "l2.mix.left.q": t["l2.mix.left.q"][:-1]}, "cpu", torch.float32)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_trace_replay_program(tmp_path, device, dtype):
    """The command-line replay: a checkpoint folder in, steps on standard input, logits in files."""
    cfg = config((gla(), None), (latent(window=20), None), (parallel(), None))
    t = weights_for(cfg, seed=31)
    save_checkpoint(str(tmp_path), cfg, {k: v.bfloat16() for k, v in t.items()})
    a, b = [3, 9, 27, 81, 5, 15], list(range(70))
    want = {r: oracle.forward(cfg, t, v)[0] for r, v in (("a", a), ("b", b))}
    steps = [([("a", a[:4], [0, 3]), ("b", b[:66], [])], []), ([("b", b[66:67], [])], []), ([("a", a[4:], [1]), ("b", b[67:], [2, 0])], ["a", "b"]),
             ([("c", a, [5])], ["c"])]
    text = "".join(json.dumps({"step": i, "entries": [{"id": r, "tokens": k, "want": w} for r, k, w in e], "end": end}) + "\n"
                   for i, (e, end) in enumerate(steps))
    exe = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([exe, "--model", str(tmp_path), "--dtype", str(dtype).split(".")[1], "--out", str(out), "--max-tokens", "192",
                        "--device", device], input=text, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert r.stdout.split() == [w for i in range(4) for w in ("done", str(i))]
    assert sorted(p.name for p in out.iterdir()) == ["0.f32", "2.f32", "3.f32"]
    load = lambda i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy())
    noise = functools.cache(lambda r: rounding_noise(cfg, t, a if r == "a" else b)[0])
    for i, rows in ((0, [("a", 0), ("a", 3)]), (2, [("a", 5), ("b", 69), ("b", 67)]), (3, [("a", 5)])):
        check_rows(load(i), torch.stack([want[r][k] for r, k in rows]), lambda: torch.stack([noise(r)[k] for r, k in rows]), dtype, i)
