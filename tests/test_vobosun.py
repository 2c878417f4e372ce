"""Vobosun against the plain implementation in ``vobosun_oracle``: every mechanism alone, then whole models through the engine's
own step (portions, mixed batches, reused pages and slots, far keys, long decoding) and greedy generation through its scheduler.
CPU runs take the package's PyTorch operations in fp32; GPU runs take the kernels in fp32 and bf16."""

import copy
import functools
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import vobosun_oracle as oracle  # noqa: E402
from modular_b200 import ops
from modular_b200.entrypoints.llm import LLM
from modular_b200.entrypoints.trace import TraceSession
from modular_b200.models.vobosun import VobosunConfig, VobosunWeights, xielu_factors
from modular_b200.nn.general_delta import GeneralDelta, GeneralDeltaConfig
from modular_b200.nn.moe import ScoreRouter, ScoreRouterConfig, expert_mlp, gated_mlp
from modular_b200.nn.residual import tanh_seam
from modular_b200.nn.rotary_embedding import RopeScaling, cos_sin_table
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


def part(t, prefix):
    return {k[len(prefix):]: v for k, v in t.items() if k.startswith(prefix)}


# ---------------------------------------------------------------------------------- configurations and weights
def dense(ff=104):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=3, identity=2, groups=(2, 1), ff=72, shared=56):
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router, **({"shared": {"ff": shared}} if shared else {})}


def attention(heads=6, kv_heads=2, dim=40, vdim=24, dims=32, base=3000.0, factor=4.0, scale=None):
    rot = {"base": base, "dims": dims, "scaling": {"factor": factor}}
    return {"type": "attention", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=rot, scale=scale or dim ** -0.5)}


def delta(heads=3, dim=24):
    return {"type": "general_delta", "mixer": dict(heads=heads, dim=dim)}


def config(*layers, width=104, vocab=190, eps=1e-5):
    """Layers are mixers (followed by a dense feed-forward), pairs (mixer, feed-forward or None), or the number of a layer whose
    weights are used again."""
    out = []
    for l in layers:
        if isinstance(l, int):
            out.append({**copy.deepcopy(out[l]), "weights_of": l})
            continue
        m, ff = l if isinstance(l, tuple) else (l, dense())
        out.append({**copy.deepcopy(m), "mlp": copy.deepcopy(ff)})
    return {"architecture": "Vobosun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out}


def weights_for(cfg, seed=0, rank=20, dtype=torch.bfloat16):
    """Random tensors of a checkpoint, rounded to ``dtype``; scores, rates and shifts such that a wrong key or state shows."""
    g = torch.Generator().manual_seed(seed)
    c, t = VobosunConfig.from_hf(cfg), {}
    for name, shape in c.tensor_shapes({i: rank for i in c.of_type("general_delta")}).items():
        v, leaf = torch.randn(shape, generator=g), name.rsplit(".", 1)[-1]
        if leaf == "alpha":
            v = 0.8 + 0.2 * v
        elif leaf == "b":
            v = 0.3 * v
        elif leaf == "shift":
            v = 0.5 + 0.4 * v
        elif leaf == "correction":
            v = 0.3 * v - 0.4                                    # choice scores on both sides of zero
        elif "norm" in leaf:
            v = 1.0 + 0.2 * v
        elif name != "embed" and leaf not in ("w0", "act"):
            v = v * shape[-1] ** -0.5 * (2.0 if leaf in ("q", "router", "w2") else 1.0)
        t[name] = v
    return {k: v.to(dtype).float() for k, v in t.items()}


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


# ---------------------------------------------------------------------------------- seams and activations
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("width", [64, 203, 1336, 5000])
def test_tanh_seam(width, device, dtype):
    """Embedding, a branch, weighted experts with identity experts and a shared expert, some rows only."""
    T, V, pad, k = 7, 20, (width + 7) // 8 * 8, 3
    r = lambda i, *s: torch.nn.functional.pad(rand(*s, width, seed=width + i), (0, pad - width)).to(dtype)
    table, a, e, own = r(0, V), 2.0 * r(1, T), r(2, T * k), r(3, T)
    nu, n1 = ((alpha, r(i, 1)[0], r(i + 1, 1)[0]) for alpha, i in ((0.7, 4), (-1.6, 6)))
    ids = torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(0))
    inverse = torch.randperm(T * k, generator=torch.Generator().manual_seed(1)).view(T, k).int()
    inverse[2, 1] = inverse[4] = -1
    pw = torch.rand(T, k, generator=torch.Generator().manual_seed(2))
    D, d = (lambda t: t.to(device)), (lambda t: t[..., :width].double())
    N = lambda n: (n[0], D(n[1]), D(n[2]))
    norm = lambda y, n: oracle.dynamic_tanh(y, n[0], d(n[1]), d(n[2]))
    x, out = torch.empty(T, pad, device=device), torch.empty(T, pad, dtype=dtype, device=device)
    tanh_seam(ids=D(ids), table=D(table), scale=0.3, x_out=x, norm1=N(n1), n1=out)
    h = 0.3 * d(table)[ids]
    assert rel(x[:, :width], h) < 1e-6 and rel(out[:, :width], norm(h, n1)) < TOL[dtype]
    tanh_seam(x=x, x_out=x, a=D(a), norm_u=N(nu), norm1=N(n1), n1=out)
    h = h + norm(d(a), nu)
    assert rel(x[:, :width], h) < 2e-6 and rel(out[:, :width], norm(h, n1)) < TOL[dtype]
    rows_of = torch.where((inverse < 0).unsqueeze(2), d(own).unsqueeze(1), d(e)[inverse.clamp(min=0).long()])
    u = (rows_of * pw.double().unsqueeze(2)).sum(1)
    kw = dict(e=D(e), inverse=D(inverse), pair_w=D(pw), norm_u=N(nu))
    y = x.clone()
    tanh_seam(x=y, x_out=y, self_rows=D(own), **kw)                                        # identity experts
    assert rel(y[:, :width], h + norm(u, nu)) < 2e-6 and (y[:, width:] == 0).all()
    y = x.clone()
    tanh_seam(x=y, x_out=y, **kw)                                                          # pairs without a row count nothing
    assert rel(y[:, :width], h + norm((torch.where((inverse < 0).unsqueeze(2), 0.0, rows_of) * pw.double().unsqueeze(2)).sum(1), nu)) < 2e-6
    rows, few, before = i32(6, 0, 6, 4), torch.empty(4, pad, dtype=dtype, device=device), x.clone()
    tanh_seam(x=x, rows=D(rows), a=D(a), self_rows=D(own), norm1=N(n1), n1=few, **kw)      # a shared expert beside the others
    h = h + norm(u + d(a), nu)
    assert torch.equal(x, before) and rel(few[:, :width], norm(h, n1)[rows.long()]) < TOL[dtype] and (few[:, width:] == 0).all()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("lens,steps", [(STEP_LENS, STEPS), ({"a": 700, "b": 75}, ([("a", 603), ("b", 1)], [("b", 2), ("a", 1)], [("a", 96), ("b", 72)])),
                                        ({"a": 4110, "b": 3001}, ([("b", 2999), ("a", 2001)], [("a", 2109), ("b", 2)]))], ids=["short", "long", "longer"])
def test_token_shift(lens, steps, device, dtype):
    """Two sequences in portions beside each other, in slots that held something else; the rows before a portion, a tile of rows and
    the first token; the update goes to a second buffer."""
    W = 40 if max(lens.values()) > 100 else 203
    pad = (W + 7) // 8 * 8
    p = lambda t: torch.nn.functional.pad(t, (0, pad - W))
    r = lambda i: p(rand(W, seed=i)).to(dtype)
    nu, n1, mix = (0.6, r(1), r(2)), (-0.9, r(3), r(4)), r(5)
    d = lambda t: t[..., :W].double()
    N, D = (lambda n: (n[0], n[1].to(device), n[2].to(device))), (lambda t: t.to(device))
    x = {s: p(rand(n, W, seed=n)) for s, n in lens.items()}
    u = {s: p(rand(n, W, seed=n + 1)).to(dtype) for s, n in lens.items()}
    norm = lambda y, n: oracle.dynamic_tanh(y, n[0], d(n[1]), d(n[2]))
    new = {s: d(x[s]) + norm(d(u[s]), nu) for s in lens}
    want = {s: oracle.token_shift(norm(new[s], n1), d(mix)) for s in lens}
    prev, slot, got = torch.full((5, pad), 7.0, device=device), {"a": 3, "b": 1}, {"a": [], "b": []}
    for rows, qs, ql, kl in two_sequences(lens, steps):
        cat = lambda t: D(torch.cat([t[s][lo:hi] for s, lo, hi in rows]))
        xin, before = cat(x), cat(x)
        xout, h = torch.empty_like(xin), torch.empty(xin.shape, dtype=dtype, device=device)
        tanh_seam(x=xin, x_out=xout, a=cat(u), norm_u=N(nu), norm1=N(n1), n1=h, shift=D(mix), prev=prev,
                  state_idx=D(i32(*[slot[s] for s, _, _ in rows])), q_start=D(qs), q_len=D(ql), kv_len=D(kl))
        assert torch.equal(xin, before) and rel(xout[:, :W], torch.cat([new[s][lo:hi] for s, lo, hi in rows])) < 2e-6
        assert (h[:, W:] == 0).all()
        for (s, lo, hi), o in zip(rows, qs.tolist()):
            got[s].append(h[o: o + hi - lo, :W])
    for s in lens:
        y = torch.cat(got[s])
        assert rel(y, want[s]) < TOL[dtype], s
        err = (y.double().cpu() - want[s]).abs().amax(1)
        assert err.max() < (1e-5 if dtype == torch.float32 else 0.05), (s, int(err.argmax()))
        assert rel(prev[slot[s], :W], norm(new[s], n1)[-1]) < 3e-6
    assert (prev[[0, 2, 4]] == 7.0).all()


@pytest.mark.parametrize("device,dtype", RUNS)
def test_token_shift_without_a_slot(device, dtype):
    """Sequences with slot -1 start from zeros and keep nothing (the dummies of a padded decode batch)."""
    W, T = 64, 5
    r = lambda i, *s: rand(*s, seed=i).to(device)
    x, mix, prev = r(1, T, W), r(2, W).to(dtype), torch.full((2, W), 3.0, device=device)
    n1 = (0.5, torch.ones(W, dtype=dtype, device=device), torch.zeros(W, dtype=dtype, device=device))
    for lens in ((1,) * T, (3, 2)):
        h, y, ql = torch.empty(T, W, dtype=dtype, device=device), torch.empty_like(x), i32(*lens).to(device)
        tanh_seam(x=x, x_out=y, norm1=n1, n1=h, shift=mix, prev=prev, state_idx=torch.full_like(ql, -1), q_start=(torch.cumsum(ql, 0) - ql).int(),
                  q_len=ql, kv_len=ql + 9)
        want = torch.cat([oracle.token_shift(torch.tanh(0.5 * v), mix.double().cpu()) for v in x.double().cpu().split(lens)])
        assert rel(h, want) < TOL[dtype] and (prev == 3.0).all() and torch.equal(x, y)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_activations(device, dtype):
    z = torch.cat([torch.linspace(-30.0, 30.0, 2000), torch.linspace(-0.5, 0.5, 1000), torch.tensor([0.0, -1e-3, 1e-3, -1e-6, 1e-6, -80.0, 80.0, -0.25])])
    z = z.to(dtype)
    for act in ((0.3, -0.7), (-2.0, 1.5), (30.0, -40.0)):
        up, down = xielu_factors(torch.tensor(act))
        assert up == pytest.approx(math.log1p(math.exp(act[0]))) and down == pytest.approx(0.5 + math.log1p(math.exp(act[1])))
        want = oracle.xielu(z.double(), *torch.tensor(act, dtype=torch.float64))
        got = ops.xielu(z.clone().view(8, -1).to(device), up, down).flatten().double().cpu()
        assert ((got - want).abs() <= (1e-5 if dtype == torch.float32 else 5e-3) * want.abs() + 1e-6).all()
    wide = torch.zeros(8, z.numel() // 8 + 16, dtype=dtype)
    wide[:, 8:-8] = z.view(8, -1)
    wide = wide.to(device)
    ops.tanh(wide[:, 8:-8])                                                                # a column range
    assert ((wide[:, 8:-8].double().cpu() - torch.tanh(z.double()).view(8, -1)).abs().max() < (2e-6 if dtype == torch.float32 else 4e-3))
    assert (wide[:, :8] == 0).all() and (wide[:, -8:] == 0).all()


# ---------------------------------------------------------------------------------- softmax attention
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("hd,dim,dims,factor", [(64, 40, 32, 1.0), (64, 64, 64, 3.0), (128, 100, 20, 8.0), (128, 72, 0, 1.0), (64, 24, 2, 0.5), (168, 168, 160, 2.0),
                                                (128, 128, 48, 2.0)])
def test_biased_and_rotated_heads(hd, dim, dims, factor, device, dtype):
    """Biases on queries, keys and values, rotation of pairs half the rotated width apart, the store into shuffled pages."""
    T, H, KH, page, first, base = 9, 5, 2, 64, 300, 700.0
    cs = cos_sin_table(dims, first + T, base, RopeScaling("linear", factor), device) if dims else None
    x, bias = torch.zeros(T, H + 2 * KH, hd), torch.zeros(H + 2 * KH, hd)
    x[..., :dim], bias[..., :dim] = rand(T, H + 2 * KH, dim, seed=dims), rand(H + 2 * KH, dim, seed=dims + 1)
    x = x.to(dtype)
    y = x.reshape(T, -1).clone().to(device)
    kv = torch.full((8, 2, 3, KH, page, hd), 5.0, dtype=dtype, device=device)
    slots = torch.randperm(8 * page, generator=torch.Generator().manual_seed(1))[:T]
    slots[4] = -1
    block_prep(y, H, H * hd, (H + KH) * hd, KH, dims, torch.arange(first, first + T, dtype=torch.int32, device=device), cs, slots.to(device), kv, 1,
               halves=True, bias=bias.flatten().to(device))
    want = x.double() + bias.double()
    if dims:
        want[:, : H + KH] = oracle.rotate(want[:, : H + KH], {"base": base, "dims": dims, "scaling": {"factor": factor}}, first)
    assert rel(y.view(T, -1, hd)[:, :H], want[:, :H]) < TOL[dtype]
    keep = [t for t in range(T) if t != 4]
    for i, lo in ((0, H), (1, H + KH)):
        rows = kv[:, i, 1].transpose(1, 2).reshape(-1, KH, hd)
        assert rel(rows[slots[keep].to(device)], want[keep, lo: lo + KH]) < TOL[dtype]
        others = torch.ones(8 * page, dtype=torch.bool)
        others[slots[keep]] = False
        assert (rows[others.to(device)] == 5.0).all()
    assert (kv[:, :, [0, 2]] == 5.0).all()


def run_attention(m, device, dtype, pieces, T, page=64):
    cfg = config(m)
    W, c, t = cfg["width"], VobosunConfig.from_hf(cfg), weights_for(cfg, seed=1)
    a, hd = c.attention(0), c.head_width
    mix = WindowAttention(a, part(t, "l0.mix."), hd, W, device, dtype)
    mix.w_in = mix.w_in.to(device, dtype)
    h = rand(T, W, seed=2).to(dtype)
    want = oracle.attention_mixer(h.double(), double(t), "l0.mix.", m["mixer"])
    bt, pages, slots = paged(T, page)
    kv = torch.full((pages, 2, 2, a.kv_heads + 1, page, hd), 4.0, dtype=dtype, device=device)
    cs = cos_sin_table(a.rot_dims, T, a.rope_base, a.rope_scaling, device)
    D, got, at = (lambda *v: i32(*v).to(device)), [], 0
    for n in pieces:
        plan = tensor_core_plan(a.group_pad, hd, dtype, page, D(0), D(n), n, n == 1)
        px = ops.linear(h[at: at + n].to(device), mix.w_in)
        mix.prep(px, torch.arange(at, at + n, dtype=torch.int32, device=device), cs, slots[at: at + n].to(device), kv, 1)
        o = mix(px[:, : mix.k_off], kv, 1, bt.to(device), D(0), D(n), D(at + n), plan)
        got.append(ops.linear(o, mix.w_o)[:, :W])
        at += n
    return torch.cat(got), want


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("m", [attention(), attention(1, 1, 8, 8, 2), attention(5, 1, 72, 128, 72, factor=1.0), attention(6, 3, 160, 40, 100),
                               attention(34, 2, 16, 32, 8), attention(8, 8, 64, 64, 16, base=1e6, scale=0.3)],
                         ids=["odd", "small", "wide", "wide head", "many heads", "no groups"])
def test_attention_mixer(m, device, dtype):
    for pieces in ((85, 2, 61, 1, 1), (150,)):
        got, want = run_attention(m, device, dtype, pieces, 150)
        assert rel(got, want) < TOL[dtype]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("heads,kv_heads,hd", [(8, 1, 64), (16, 4, 128), (3, 3, 64)])
@pytest.mark.parametrize("place", [0, 1, 62, 63, 64, 128, 255])
def test_one_far_key(place, heads, kv_heads, hd, device, dtype):
    """One key among hundreds stands out for every query: it is found from its own position on, whatever page it lies in, in
    prompts, from portions and from decoding, and not before."""
    page, T = 64, 600
    k, v = (rand(T, kv_heads, hd, seed=s) for s in (place, place + 1))
    q = 0.05 * rand(T, heads, hd, seed=place + 2)
    k *= 0.05
    k[place, :, 3] = 6.0
    q[:, :, 3] = 6.0
    k, v, q = (x.to(dtype) for x in (k, v, q))
    want = oracle.attention(q.double(), k.double(), v.double(), 0.5)
    assert (want[place:] - v[place].double().repeat_interleave(heads // kv_heads, 0)).abs().max() < 1e-3
    bt, pages, slots = paged(T, page, seed=place)
    kv = torch.zeros(2, pages * page, kv_heads, hd, dtype=dtype)
    kv[0, slots], kv[1, slots] = k, v
    kv = kv.view(2, pages, page, kv_heads, hd).permute(1, 0, 3, 2, 4).unsqueeze(2).contiguous().to(device)
    D = lambda *x: i32(*x).to(device)
    spans = [(0, T), (max(place - 70, 0), place + 3), (T - 2, T), (T - 1, T), (place, place + 1), (place, place + 2)]
    spans += [(place - 1, place), (place - 1, place + 1)] if place else []
    for lo, hi in spans:
        plan = tensor_core_plan(heads // kv_heads if heads // kv_heads != 3 else 4, hd, dtype, page, D(0), D(hi - lo), hi - lo, hi - lo == 1)
        got = window_attention(q[lo:hi].reshape(hi - lo, -1).to(device), kv, 0, bt.to(device), D(0), D(hi - lo), D(hi), heads, kv_heads, 0.5, plan=plan)
        err = (got.double().cpu().view(hi - lo, heads, hd) - want[lo:hi]).abs().amax((1, 2))
        assert err.max() < (1e-4 if dtype == torch.float32 else 5e-2), (lo, hi, lo + int(err.argmax()))


# ---------------------------------------------------------------------------------- generalized delta rule
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,d,rank", [(3, 24, 20), (1, 8, 1), (5, 64, 72), (2, 128, 16), (4, 9, 8), (2, 100, 40), (1, 300, 16), (2, 200, 130), (36, 32, 4)])
def test_general_delta_mixer(H, d, rank, device, dtype):
    """Two sequences in portions beside each other, in slots that held something else before."""
    W = 104
    cfg = config(delta(H, d), width=W)
    t, c = weights_for(cfg, seed=d, rank=rank), GeneralDeltaConfig(H, d, rank, 1e-5)
    mix, w = GeneralDelta(c, part(t, "l0.mix."), W, device, dtype), double(t)
    h = {s: rand(n, W, seed=n).to(dtype) for s, n in STEP_LENS.items()}
    want = {s: oracle.general_delta_mixer(x.double(), w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5) for s, x in h.items()}
    state = torch.full((5, *c.state_shapes()["gdelta"]), 3.0, device=device)
    slot, got = {"a": 3, "b": 1}, {"a": [], "b": []}
    for rows, qs, ql, kl in two_sequences(STEP_LENS, STEPS):
        x = torch.cat([h[s][lo:hi] for s, lo, hi in rows]).to(device)
        y = mix(x, ops.linear, state, i32(*[slot[s] for s, _, _ in rows]).to(device), qs.to(device), ql.to(device), kl.to(device),
                bool((ql == 1).all()))
        for (s, lo, hi), o in zip(rows, qs.tolist()):
            got[s].append(y[o: o + hi - lo, :W])
    for s in h:
        y = torch.cat(got[s])
        if dtype == torch.float32:
            assert rel(y, want[s]) < TOL[dtype], s
        else:                                      # the norm enlarges what rounding does to a head that gives almost nothing
            err = (y.double().cpu() - want[s]).pow(2).mean(1).sqrt() / want[s].pow(2).mean().sqrt()
            assert err.median() < TOL[dtype] and (err < 2 * TOL[dtype]).double().mean() > 0.95, s
    assert (state[[0, 2, 4]] == 3.0).all()                                                 # nobody else's slot was written


def bare_delta(H, d, device, dtype):
    zero = lambda *s: torch.zeros(*s)
    t = {n: zero(H * d, 8) for n in "rkvga"}
    t.update({"a.b": zero(H * d), "w1": zero(4, 8), "w2": zero(H * d, 4), "w0": zero(H * d), "norm": torch.ones(H * d), "o": zero(8, H * d)})
    return GeneralDelta(GeneralDeltaConfig(H, d, 4, 1e-5), t, 64, device, dtype)


def drive(mix, r, k, v, a, z, pieces, state, device):
    """Projections [T, H, d] of one sequence through the mixer in portions; heads without the gate, [T, H, d]."""
    T, H, d = r.shape
    px = torch.zeros(T, mix.w_off + 64, dtype=r.dtype)
    for off, x in ((0, r), (mix.k_off, k), (mix.v_off, v), (mix.a_off, a)):
        px[:, off: off + H * d] = x.reshape(T, -1)
    px[:, mix.g_off: mix.a_off] = 40.0                                                     # sigmoid(40) = 1
    D, got, at = (lambda *x: i32(*x).to(device)), [], 0
    for n in pieces:
        out = torch.empty(n, H * d, dtype=r.dtype, device=device)
        mix.mix(px[at: at + n].to(device), z[at: at + n].to(device), out, state, D(0), D(0), D(n), D(at + n), n == 1)
        got.append(out.double().cpu())
        at += n
    return torch.cat(got).view(T, H, d)


def unit_rms(o, eps=1e-5):
    return o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("gap", [1, 2, 15, 16, 17, 33, 300])
def test_general_delta_remembers_and_forgets(gap, device, dtype):
    """One key far back that a query asks for after ``gap`` slow decays; in between the same key is written again with another value,
    in one head with removal, in the other without."""
    H, d, T = 2, 32, 340
    r, k, v = (0.02 * rand(T, H, d, seed=gap + s) for s in range(3))
    z = torch.full((T, H * d), -9.0)                                                       # decays close to one
    key = torch.randn(H, d, generator=torch.Generator().manual_seed(5))
    k[20], v[20], r[20 + gap] = key, 3.0 * rand(H, d, seed=6), key
    a = torch.full((T, H, d), -30.0)
    if gap > 1:
        k[20 + gap - 1], v[20 + gap - 1] = 0.5 * key, rand(H, d, seed=7)
        a[20 + gap - 1, 0] = 30.0                                                          # head 0 forgets the first value
    r, k, v, a = (x.to(dtype) for x in (r, k, v, a))
    decay = torch.exp(-math.exp(-0.5) * oracle.sigmoid(z.double())).view(T, H, d)
    rate = oracle.sigmoid(a.double())
    want, S = oracle.general_delta_scan(r.double(), k.double(), v.double(), decay, rate)
    want = unit_rms(want)
    if gap > 1:                                                                            # the two heads hold different things now
        first, second = (unit_rms(x[None])[0] for x in (v[20].double(), v[20 + gap - 1].double()))
        cos = lambda x, y: float((x * y).sum() / x.norm() / y.norm())
        assert cos(want[20 + gap, 0], second[0]) > 0.95 and cos(want[20 + gap, 1], first[1]) > 0.9
    mix = bare_delta(H, d, device, dtype)
    for pieces in ((T,), (20 + gap, T - 20 - gap), (21, 1, gap - 1, T - 21 - gap) if gap > 1 else (21, 1, T - 22), (21 + gap, 2, T - 23 - gap)):
        state = torch.full((1, *mix.cfg.state_shapes()["gdelta"]), 9.0, device=device)
        got = drive(mix, r, k, v, a, z, pieces, state, device)
        assert rel(got[20 + gap], want[20 + gap]) < TOL[dtype], pieces
        assert rel(got, want) < 2 * TOL[dtype], pieces
        assert rel(state[0, :, :, :d].transpose(1, 2), S) < 2e-5


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,d", [(2, 8), (3, 64), (5, 96), (2, 128), (1, 200), (1, 512)])
def test_general_delta_kernel_keeps_fp32(H, d, dtype):
    """States and outputs before the norm against the plain recurrence in float64 on the same projections: sequences that begin, go
    on, or have one token; decays and removal rates from none to all within a head."""
    from modular_b200._native import lib

    lens, old, slots = [70, 1, 33, 2, 40, 17], [0, 5, 64, 7, 130, 1], [3, 0, 5, -1, 1, 6]
    T, pad = sum(lens), next(n for n in (32, 64, 96, 128, 192, 256, 512) if d <= n)
    x = rand(T, 5 * H * d, seed=d).to(dtype)
    x[:, 4 * H * d:] *= 6.0
    z, zb, ab, w = 6.0 * rand(T, H * d, seed=2), rand(H * d, seed=3), rand(H * d, seed=4), torch.ones(H * d, dtype=dtype)
    state = torch.zeros(8, H, d, pad)
    state[..., :d] = rand(8, H, d, d, seed=5)
    ql = i32(*lens)
    kl, qs = ql + i32(*old), (torch.cumsum(ql, 0) - ql).int()
    st, o, out = state.cuda(), torch.empty(T, H, d, device="cuda"), torch.empty(T, H * d, dtype=dtype, device="cuda")
    gx = x.cuda()
    lib().general_delta(gx, 0, H * d, 2 * H * d, 4 * H * d, ab.cuda(), z.cuda(), zb.cuda(), gx[:, 3 * H * d: 4 * H * d], w.cuda(), 1e-5, d,
                        torch.empty(T * H * (4 * pad + 4), device="cuda"), o, out, st, i32(*slots).cuda(), qs.cuda(), ql.cuda(), kl.cuda(), H, d, d,
                        False)
    decay = torch.exp(-math.exp(-0.5) * oracle.sigmoid(z.double() + zb.double())).view(T, H, d)
    rate = oracle.sigmoid(x[:, 4 * H * d:].double() + ab.double()).view(T, H, d)
    r, k, v, _, _ = (y.double().view(T, H, d) for y in x.split(H * d, 1))
    for i, n in enumerate(lens):
        t = slice(int(qs[i]), int(qs[i]) + n)
        S0 = state[slots[i], :, :, :d].transpose(1, 2).double() if slots[i] >= 0 and old[i] else None
        want, S = oracle.general_delta_scan(r[t], k[t], v[t], decay[t], rate[t], S0)
        assert rel(o[t], want) < 1e-5, i
        if slots[i] >= 0:
            assert rel(st[slots[i], :, :, :d].transpose(1, 2), S) < 1e-5 and (st[slots[i], :, :, d:] == 0).all()
    assert torch.equal(st[[2, 4, 7]].cpu(), state[[2, 4, 7]])


@pytest.mark.parametrize("device,dtype", RUNS)
def test_general_delta_without_a_slot(device, dtype):
    W = 104
    cfg = config(delta(), width=W)
    t, D = weights_for(cfg), lambda *v: i32(*v).to(device)
    c = GeneralDeltaConfig(3, 24, 20, 1e-5)
    mix, w, state = GeneralDelta(c, part(t, "l0.mix."), W, device, dtype), double(t), torch.ones((2, *c.state_shapes()["gdelta"]), device=device)
    for lens in ((1, 1), (70, 3)):
        x = rand(sum(lens), W).to(device, dtype)
        y = mix(x, ops.linear, state, D(-1, -1), D(0, lens[0]), D(*lens), D(lens[0], 99), lens == (1, 1))
        for lo, hi in ((0, lens[0]), (lens[0], sum(lens))):
            want = oracle.general_delta_mixer(x[lo: hi].cpu().double(), w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5)
            assert rel(y[lo: hi, :W], want) < TOL[dtype]
    assert (state == 1).all()


# ---------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("ff", [moe(), moe(8, 4, 0, None, 24, 0), moe(1, 1, 0, (1, 1), 64, 8), moe(1, 3, 3, (2, 2), 64, 72), moe(38, 7, 2, (5, 2), 16, 200),
                                moe(61, 8, 3, None, 8), moe(96, 3, 0, (96, 40), 8), moe(250, 10, 10, (4, 2), 8), moe(12, 16, 4, (4, 4), 8),
                                moe(3, 2, 9, (3, 2), 24)],
                         ids=lambda f: "-".join(str(f["router"].get(k, 0)) for k in ("experts", "top", "identity")))
def test_router_experts_identity_and_shared(ff, device, dtype):
    """The choice (choice scores on both sides of zero), the weights, the order of the rows, and the whole sum through the seam."""
    W, T = 96, 77
    cfg = config((delta(), ff), width=W)
    t, c = weights_for(cfg, seed=2), VobosunConfig.from_hf(cfg).router(0)
    t["l0.mlp.router"] *= 4.0
    r, w, E, top = ff["router"], double(t), c.experts, c.top
    x = rand(T, W, seed=1).to(dtype)
    router = ScoreRouter(c, t["l0.mlp.router"], t["l0.mlp.correction"], W, device, dtype)
    rows, offsets, inverse, weights = router.route(x.to(device), torch.zeros(E, dtype=torch.int32, device=device))
    inv, off, wt = inverse.cpu().long(), offsets.cpu().tolist(), weights.cpu()
    placed = sorted(p for p in inv.flatten().tolist() if p >= 0)
    assert placed == list(range(off[-1])) and off[0] == 0 and (inv >= -1).all()
    at, slot = torch.nonzero(inv >= 0, as_tuple=True)
    assert torch.equal(rows.cpu()[inv[at, slot]], x[at])
    s, clear = oracle.router_scores(x.double(), w, "l0.mlp."), []
    for i in range(T):
        if oracle.choice_margin(s[i], w["l0.mlp.correction"], r) < 1e-4:
            continue
        clear.append(i)
        chosen = oracle.choose(s[i], w["l0.mlp.correction"], r)
        mine = [next(e for e in range(E) if off[e] <= p < off[e + 1]) for p in inv[i].tolist() if p >= 0]
        assert sorted(mine) == sorted(e for e in chosen if e < E)
        total = sum(float(s[i, e]) for e in chosen)
        got = [(float(wt[i, j]), p) for j, p in enumerate(inv[i].tolist())]
        for e, (g, _) in zip(sorted(mine), sorted(((g, p) for g, p in got if p >= 0), key=lambda v: v[1])):
            assert g == pytest.approx(float(s[i, e]) / total, rel=1e-4, abs=1e-6)
        assert sum(g for g, p in got if p < 0) == pytest.approx(sum(float(s[i, e]) for e in chosen if e >= E) / total, rel=1e-4, abs=1e-6)
    assert len(clear) > T // 2 and (not c.identity or (inv < 0).any())
    F = ff["expert"]["ff"]
    pad = max(64, F) - F
    gu = torch.stack([torch.cat([t[f"l0.mlp.e{e}.gate"], t[f"l0.mlp.e{e}.up"]]) for e in range(E)])
    gu = torch.nn.functional.pad(gu.view(E, 2, F, W), (0, 0, 0, pad)).reshape(E, -1, W).to(device, dtype)
    dn = torch.nn.functional.pad(torch.stack([t[f"l0.mlp.e{e}.down"] for e in range(E)]), (0, pad)).to(device, dtype)
    xd = x.to(device)
    branch = dict(e=expert_mlp(rows, offsets, gu, dn, T), inverse=inverse, pair_w=weights, self_rows=xd if c.identity else None)
    if ff.get("shared"):
        n = "l0.mlp.shared."
        F = ff["shared"]["ff"]
        p = lambda m: torch.nn.functional.pad(m, (0, 0, 0, max(64, F) - F))
        branch["a"] = gated_mlp(xd, torch.cat([p(t[n + "gate"]), p(t[n + "up"])]).to(device, dtype),
                                torch.nn.functional.pad(t[n + "down"], (0, max(64, F) - F)).to(device, dtype))
    one = (0.01, torch.full((W,), 128.0, dtype=dtype, device=device), torch.zeros(W, dtype=dtype, device=device))       # nearly linear
    y = torch.zeros(T, W, device=device)
    tanh_seam(x=y, x_out=y, norm_u=one, **branch)
    want = oracle.dynamic_tanh(oracle.moe(x.double(), w, "l0.mlp.", ff), 0.01, 128.0, 0.0)
    err = (y.double().cpu() - want).pow(2).mean(1).sqrt() / want.pow(2).mean().sqrt()
    assert err[clear].max() < TOL[dtype]


def test_router_config_checks():
    for bad in (dict(experts=6, top=2, identity=1, groups=2), dict(experts=4, top=4, identity=2, groups=2), dict(experts=6, top=2, groups=3, keep=4),
                dict(experts=0, top=1, identity=2), dict(experts=1000, top=2, identity=25)):
        with pytest.raises(ValueError):
            ScoreRouterConfig(**bad)
    assert ScoreRouterConfig(5, 3, 2, 1, identity=1).candidates == 6


# ---------------------------------------------------------------------------------- whole models
MIXED = config(attention(), (delta(), moe()), (attention(4, 4, 24, 56, 16, 700.0, 1.0), moe(5, 2, 0, None, 40, 0)), 1, (delta(2, 72), None),
               (attention(heads=7, kv_heads=1, dim=56, vdim=40, dims=56, factor=0.5), None), (delta(5, 16), dense(64)), 0, 1)


def clear_choices(t, dtype):
    """Runs that round would choose other experts where two choices are close, and such a token changes all that follow: their
    experts depend on the corrections (the choice itself has a test of its own, and fp32 runs choose by token)."""
    return t if dtype == torch.float32 else {k: (20.0 * v).bfloat16().float() if k.endswith("correction") else v for k, v in t.items()}


@functools.cache
def mixed_reference(dtype):
    t = clear_choices(weights_for(MIXED), dtype)
    draw = lambda n, s: torch.randint(0, MIXED["vocab"], (n,), generator=torch.Generator().manual_seed(s)).tolist()
    out = {}
    for r, toks in (("a", draw(260, 3)), ("b", draw(140, 4))):
        out[r] = (toks, *oracle.forward(MIXED, t, toks), functools.cache(lambda toks=toks: rounding_noise(MIXED, t, toks)))
    return t, out


@pytest.fixture(scope="module")
def mixed_model():
    return mixed_reference


def engine(cfg, t, device, dtype, tokens=512, page=64, batch=4, **kw):
    c = VobosunConfig.from_hf(cfg)
    args = dict(max_length=tokens, max_batch_size=batch, max_batch_input_tokens=tokens, page_size=page,
                num_kv_pages=-(-tokens // page) + 1, enable_prefix_caching=False, max_logit_rows=tokens,
                enable_overlap_scheduler=False, graph_batch_sizes=[1, 4])
    args.update(kw)
    return LLM(c, VobosunWeights.from_state_dict(c, t, device, dtype), device=device, dtype=dtype, **args)


def rounding_noise(cfg, t, tokens, samples=2):
    """How far rounding the operands and results of matrix products to 16 bits moves the rows of the plain implementation:
    (logits, stream), the largest of some samples."""
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
        assert err.max() < 5e-4 * unit, (what, int(err.argmax()), float(err.max() / unit))
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
    assert len(stream) == len(want) == 9 and stream[0].dtype == torch.float32
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
    "whole": [[("a", 260)], [("b", 140)]],
    "token by token": [[("b", 1)]] * 140,
    "long decoding": [[("a", 20)]] + [[("a", 1)]] * 240,
    "twos": [[("a", n)] for n in cut(260, 2)],
    "page borders": [[("a", n)] for n in cut(260, 63, 1, 1, 63, 2, 62, 64)],
    "changing": [[("a", n)] for n in cut(260, 2, 3, 50, 2, 17, 5)],
    "mixed": [[("a", 100), ("b", 3)], [("b", 60), ("a", 1)], [("a", 1), ("b", 1)], [("b", 2), ("a", 90)], [("a", 1)], [("b", 74), ("a", 67)]],
    "reuse": [[("a", 160), ("b", 70)], [("b", 70), ("a", 2)], [("b#2", 2), ("a", 40)], [("a", 1), ("b#2", 1)], [("a", 57), ("b#2", 40)],
              [("b#2", 97), ("b#3", 9)], [("a#2", 110), ("b#3", 1)], [("a#2", 1), ("b#3", 1)], [("b#3", 129)], [("a#2", 149)]],
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
    config(attention()), config(delta()), config((delta(), moe())),
    config((attention(1, 1, 4, 4, 2), moe(1, 1, 1, None, 4, 4)), (delta(1, 4), None), (attention(1, 1, 4, 4, 4), dense(4)), 0, width=42, vocab=33),
    config((attention(10, 2, 104, 80, 60), moe(12, 5, 4, (4, 3), 136, 72)), delta(7, 104), width=202, vocab=98, eps=1e-3),
    config(attention(2, 2, 200, 144, 66), attention(3, 1, 32, 32, 32), delta(1, 144), width=88),
    config((delta(2, 40), moe(4, 4, 2, (2, 2), 24, 0)), (attention(), moe(9, 2, 0, (3, 1), 8, 8)), 1, 1, 0)],
    ids=["attention only", "delta only", "experts", "tiny", "wide", "wide heads", "weights used again"])
def test_other_sizes(cfg, device, dtype):
    t = clear_choices(weights_for(cfg, seed=11, rank=9), dtype)
    toks = torch.randint(0, cfg["vocab"], (150,), generator=torch.Generator().manual_seed(1)).tolist()
    want = oracle.forward(cfg, t, toks)[0]
    out = replay(engine(cfg, t, device, dtype), {"a": toks}, [[("a", n)] for n in (40, 2, 1, 1, 21, 1, 84)])
    check_rows(out["a"], want, lambda: rounding_noise(cfg, t, toks)[0], dtype)


@pytest.mark.parametrize("device,dtype", [RUNS[0], RUNS[2]])
def test_pages_of_other_sizes(device, dtype):
    """Pages that are a multiple of 64 tokens and pages that are not (no tensor-core attention then)."""
    cfg = config(attention(), delta())
    t = weights_for(cfg, seed=12)
    toks = torch.randint(0, cfg["vocab"], (260,), generator=torch.Generator().manual_seed(1)).tolist()
    want = oracle.forward(cfg, t, toks)[0]
    for page in (128, 40):
        out = replay(engine(cfg, t, device, dtype, page=page), {"a": toks}, [[("a", n)] for n in (129, 1, 1, 60, 69)])
        check_rows(out["a"], want, lambda: rounding_noise(cfg, t, toks)[0], dtype, page)


def mistakes():
    """Configurations and weights of one planted mistake each."""
    def scaling(c, t):
        c["layers"][0]["mixer"]["rot"]["scaling"]["factor"] = 5.0

    def rotated(c, t):
        c["layers"][0]["mixer"]["rot"]["dims"] = 30

    def key_bias(c, t):
        t["l2.mix.v.b"] *= 0.0

    def shift(c, t):
        t["l6.shift"] *= 0.0

    def alpha(c, t):
        t["l4.norm1b.alpha"] *= 1.1

    def rate(c, t):
        t["l1.mix.a.b"] -= 1.0

    def decay(c, t):
        t["l1.mix.w0"] *= 0.0

    def identity(c, t):
        t["l1.mlp.correction"][-2:] -= 3.0

    def groups(c, t):
        for i in (1, 3, 8):
            c["layers"][i]["mlp"]["router"]["groups"]["keep"] = 2

    def activation(c, t):
        t["l6.mlp.act"] = t["l6.mlp.act"].flip(0)

    def shared(c, t):
        t["l1.mlp.shared.down"] *= 0.0

    def sharing(c, t):
        c["layers"][7].pop("weights_of")
        t.update({k.replace("l0.", "l7.", 1): v for k, v in t.items() if k.startswith("l0.")})
        t["l7.shift"] = t["l6.shift"]

    return [scaling, rotated, key_bias, shift, alpha, rate, decay, identity, groups, activation, shared, sharing]


@pytest.mark.parametrize("plant", mistakes(), ids=lambda f: f.__name__)
def test_the_comparison_notices_mistakes(mixed_model, plant):
    """A mistake planted in the plain implementation is larger than what the whole-model tests accept."""
    t, ref = mixed_model(torch.float32)
    toks, want = ref["b"][0][:60], ref["b"][1][:60]
    c, w = copy.deepcopy(MIXED), {k: v.clone() for k, v in t.items()}
    plant(c, w)
    got = oracle.forward(c, w, toks)[0]
    err = (got - want).pow(2).mean(1).sqrt() / want.pow(2).mean().sqrt()
    assert err.max() > 20 * 5e-4 and (err > 5e-4).double().mean() > 0.2


@pytest.mark.parametrize("device,dtype", RUNS)
def test_greedy_generation(device, dtype):
    """More requests than a batch holds through the scheduler, prompts in chunks beside decoding, with preemption when the
    pool runs dry: the tokens are those of plain greedy decoding."""
    cfg = config(attention(), (delta(), moe()), (attention(heads=2, kv_heads=1), None), 1, vocab=150)
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
    cfg = config(attention(), (delta(), moe()))
    llm = engine(cfg, weights_for(cfg), "cuda:0", torch.bfloat16, max_logit_rows=0)
    sp = lambda seed: SamplingParams(temperature=1.0, top_k=20, max_new_tokens=16, ignore_eos=True, seed=seed, repetition_penalty=1.2)
    a, b = (llm.generate([[1, 2, 3], [4, 5]], [sp(s), sp(s + 1)]) for s in (5, 9))
    assert all(len(r.tokens) == 16 and 0 <= min(r.tokens) and max(r.tokens) < cfg["vocab"] for r in a + b)
    assert [r.tokens for r in a] != [r.tokens for r in b]


# ---------------------------------------------------------------------------------- configuration, command line
def test_config_checks_and_registry():
    arch = PIPELINE_REGISTRY.retrieve_architecture(MIXED)
    assert arch.name == "Vobosun" and arch.config_class is VobosunConfig
    c = VobosunConfig.from_hf(MIXED)
    again = VobosunConfig.from_hf(c.to_hf())
    assert again.layers == c.layers and PIPELINE_REGISTRY.retrieve_architecture(c.to_hf()) is arch
    assert c.of_type("attention") == (0, 2, 5, 7) and c.head_width == 64 and c.cache_heads == 4 and c.source(8) == 1
    assert [s[0] for s in c.state_specs()] == ["l0.shift", "l1.shift", "l1.gdelta", "l2.shift", "l3.shift", "l3.gdelta", "l4.shift", "l4.gdelta",
                                               "l5.shift", "l6.shift", "l6.gdelta", "l7.shift", "l8.shift", "l8.gdelta"]
    assert not any(n.startswith(("l3.", "l7.", "l8.")) for n in c.tensor_shapes())
    t = weights_for(MIXED)
    loaded = VobosunWeights.from_state_dict(c, t, "cpu", torch.float32)
    assert loaded.layers[8] is loaded.layers[1] and loaded.layers[7] is loaded.layers[0]
    other = config(delta(), delta(2))
    other["layers"][1]["weights_of"] = 0                                                   # not the same sizes
    for bad in (config(attention(5, 2)), config(attention(dims=50)), config(attention(dims=7)), config((delta(), moe(6, 5, 2, (2, 1)))),
                config((delta(), moe(6, 2, 1, (2, 1)))), other):
        with pytest.raises(ValueError):
            VobosunConfig.from_hf(bad)
    for kind in ("type", "kind"):
        bad = config(delta())
        (bad["layers"][0] if kind == "type" else bad["layers"][0]["mlp"])[kind] = "other"
        with pytest.raises(ValueError):
            VobosunConfig.from_hf(bad)
    with pytest.raises(KeyError):
        VobosunWeights.from_state_dict(c, {k: v for k, v in t.items() if k != "l2.mix.q.b"}, "cpu", torch.float32)
    with pytest.raises(ValueError):
        VobosunWeights.from_state_dict(c, {**t, "l0.mix.q": t["l0.mix.q"][:-1]}, "cpu", torch.float32)
    tiny = VobosunConfig.tiny()
    assert tiny.source(4) == 1 and tiny.is_moe(2) and tiny.layers[5]["mlp"] is None


@pytest.mark.parametrize("device,dtype", RUNS)
def test_trace_replay_program(tmp_path, device, dtype):
    """The command-line replay: a checkpoint folder in, steps on standard input, logits in files."""
    cfg = config(attention(), (delta(), None), 0)
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
