"""Vipotar against the plain implementation in ``vipotar_oracle``: every mechanism alone, then whole models through the
engine's own step (portions, mixed batches, reused pages and slots, window edges, long decoding) and greedy generation
through its scheduler. CPU runs take the package's PyTorch operations in fp32; GPU runs take the kernels in fp32 and bf16."""

import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import vipotar_oracle as oracle  # noqa: E402
from modular_b200 import ops
from modular_b200.entrypoints.llm import LLM
from modular_b200.entrypoints.trace import TraceSession
from modular_b200.models.vipotar import VipotarConfig, VipotarWeights
from modular_b200.nn.lightning_attention import LightningAttention, LightningConfig
from modular_b200.nn.parallel_block import ParallelBlock
from modular_b200.nn.residual import residual_norm
from modular_b200.nn.rotary_embedding import RopeScaling, cos_sin_table, inverse_frequencies
from modular_b200.nn.window_attention import (WindowAttention, WindowAttentionConfig, block_prep, head_width, tensor_core_plan,
                                              window_attention)
from modular_b200.pipelines.context import SamplingParams, TextContext
from modular_b200.pipelines.registry import PIPELINE_REGISTRY
from modular_b200.pipelines.weights import save_checkpoint

RUNS = [pytest.param("cpu", torch.float32, id="cpu-fp32"),
        pytest.param("cuda:0", torch.float32, id="gpu-fp32", marks=pytest.mark.gpu),
        pytest.param("cuda:0", torch.bfloat16, id="gpu-bf16", marks=pytest.mark.gpu)]
TOL = {torch.float32: 2e-4, torch.bfloat16: 3e-2}        # root mean square error over that of the expected values
YARN = dict(factor=6.0, original=200, fast=30.0, slow=1.5)


def rel(got, want):
    got, want = got.double().cpu(), want.double()
    return ((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp(min=1e-12)).item()


def i32(*v):
    return torch.tensor(v, dtype=torch.int32)


def rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def layer(heads=6, kv_heads=2, dim=40, vdim=24, window=37, dims=16, base=3000.0, scaling=None, scale=None, rheads=3, rdim=20, rvdim=28,
          decay=None, ff=72):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = scaling
    left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or 0.8 * dim ** -0.5, mask={"size": window}, rot=rot)
    right = dict(heads=rheads, dim=rdim, vdim=rvdim, decay=decay or [0.5 + 0.499 * (i + 1) / rheads for i in range(rheads)])
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(*layers, width=104, vocab=190, eps=1e-5, mult=0.6, cap=9.0, loop=None):
    return {"architecture": "Vipotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "logit_softcap": cap, "loop": loop, "layers": [copy.deepcopy(l) for l in layers]}


def weights_for(cfg, seed=0, dtype=torch.bfloat16):
    """Random tensors of a checkpoint, rounded to ``dtype``; scores and logits large enough that a wrong key shows."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    lin = lambda o, i: rnd(o, i) * i ** -0.5
    norm = lambda n: 1.0 + 0.2 * rnd(n)
    W, V = cfg["width"], cfg["vocab"]
    t = {"embed": rnd(V, W), "final.norm": norm(W), "head": 2.0 * lin(V, W)}
    if cfg["loop"]:
        t["loop.step"] = 0.5 * rnd(cfg["loop"]["times"], W)
    for i, l in enumerate(cfg["layers"]):
        a, b, p = l["mixer"]["left"], l["mixer"]["right"], f"l{i}.mix."
        t[f"l{i}.norm1"] = norm(W)
        t.update({p + "left.q": 2.0 * lin(a["heads"] * a["dim"], W), p + "left.k": lin(a["kv_heads"] * a["dim"], W),
                  p + "left.v": lin(a["kv_heads"] * a["vdim"], W), p + "left.o": lin(W, a["heads"] * a["vdim"]), p + "left.out": norm(W)})
        n = b["heads"] * b["vdim"]
        t.update({p + "right.q": lin(b["heads"] * b["dim"], W), p + "right.k": lin(b["heads"] * b["dim"], W), p + "right.v": lin(n, W),
                  p + "right.g": lin(n, W), p + "right.o": lin(W, n), p + "right.norm": norm(n), p + "right.out": norm(W)})
        if l["mlp"]:
            t.update({f"l{i}.mlp.up": lin(l["mlp"]["ff"], W), f"l{i}.mlp.down": lin(W, l["mlp"]["ff"])})
    return {k: v.to(dtype).float() for k, v in t.items()}


def engine(cfg, t, device, dtype, tokens=512, page=64, batch=4, **kw):
    c = VipotarConfig.from_hf(cfg)
    args = dict(max_length=tokens, max_batch_size=batch, max_batch_input_tokens=tokens, page_size=page,
                num_kv_pages=-(-tokens // page) + 1, enable_prefix_caching=False, max_logit_rows=tokens,
                enable_overlap_scheduler=False, graph_batch_sizes=[1, 4])
    args.update(kw)
    return LLM(c, VipotarWeights.from_state_dict(c, t, device, dtype), device=device, dtype=dtype, **args)


def paged(n_tokens, page, seed=0):
    """A block table of shuffled pages for one sequence: (table [1, n], pages in the pool, slots of every position)."""
    n = -(-n_tokens // page)
    pages = torch.randperm(n + 2, generator=torch.Generator().manual_seed(seed))[:n].int()
    pos = torch.arange(n_tokens)
    return pages.view(1, -1), n + 2, pages.long()[pos // page] * page + pos % page


# ---------------------------------------------------------------------------------- rotation, activations, seams
@pytest.mark.parametrize("dims,base,scaling", [(16, 3000.0, None), (48, 1e6, YARN), (8, 50.0, dict(factor=1.0, original=64, fast=8.0, slow=2.0)),
                                               (2, 10.0, dict(factor=3.0, original=100, fast=4.0, slow=4.0)),
                                               (64, 1e4, dict(factor=0.5, original=4096, fast=32.0, slow=1.0))])
def test_frequencies(dims, base, scaling):
    s = None if scaling is None else VipotarConfig.from_hf(config(layer(dim=64, dims=dims, base=base, scaling=scaling))).attention(0).rope_scaling
    got, amp = inverse_frequencies(dims, base, s or RopeScaling())
    want, wamp = oracle.frequencies(dims, base, scaling)
    assert np.allclose(got, want, rtol=1e-12) and abs(amp - wamp) < 1e-12
    if scaling and scaling["factor"] > 1 and dims > 2:
        assert not np.allclose(got, oracle.frequencies(dims, base)[0]) and amp > 1


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("dims", [64, 20, 6, 0])
def test_block_prep(dims, device, dtype):
    """Rotation in neighbouring pairs of queries and keys (values untouched), the store into shuffled pages, and both
    activations; a token without a slot leaves the cache alone."""
    T, H, KH, hd, page, first = 9, 4, 2, 64, 64, 300
    rot = {"dims": dims, "base": 500.0, "scaling": YARN}
    a = VipotarConfig.from_hf(config(layer(dim=64, vdim=64, dims=dims or 2, base=500.0, scaling=YARN))).attention(0)
    cs = cos_sin_table(dims, first + T, 500.0, a.rope_scaling, device) if dims else None
    cols = (H + 2 * KH) * hd
    x = rand(T, cols + 24 + 40 + 16, seed=dims).to(dtype)
    y, x = x.clone().to(device), x.double()
    kv = torch.full((8, 2, 3, KH, page, hd), 5.0, dtype=dtype, device=device)
    slots = torch.randperm(8 * page, generator=torch.Generator().manual_seed(1))[:T]
    slots[4] = -1
    block_prep(y, H, H * hd, (H + KH) * hd, KH, dims, torch.arange(first, first + T, dtype=torch.int32, device=device), cs, slots.to(device),
               kv, 1, silu=(cols + 8, 24), relu2=(cols + 40, 40))
    turn = lambda t: oracle.rotate(t, rot, first) if dims else t
    assert rel(y[:, : H * hd], turn(x[:, : H * hd].view(T, H, hd)).reshape(T, -1)) < TOL[dtype]
    k, v = turn(x[:, H * hd: (H + KH) * hd].view(T, KH, hd)), x[:, (H + KH) * hd: cols].view(T, KH, hd)
    c = kv.cpu().double()
    for t in range(T):
        if t != 4:
            pg, o = int(slots[t]) // page, int(slots[t]) % page
            assert rel(c[pg, 0, 1, :, o], k[t]) < TOL[dtype] and rel(c[pg, 1, 1, :, o], v[t]) == 0
    assert int((c != 5.0).any(-1).sum()) == 2 * KH * (T - 1) and (c[:, :, [0, 2]] == 5.0).all()
    assert rel(y[:, cols + 8: cols + 32], oracle.silu(x[:, cols + 8: cols + 32])) < TOL[dtype]
    assert rel(y[:, cols + 40:], torch.clamp(x[:, cols + 40:], min=0.0) ** 2) < TOL[dtype]
    assert rel(y[:, cols: cols + 8], x[:, cols: cols + 8]) == 0 and rel(y[:, cols + 32: cols + 40], x[:, cols + 32: cols + 40]) == 0


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("width", [64, 200, 1336])
def test_seam_with_branch_norms(width, device, dtype):
    T, V = 7, 20
    r = lambda i, *s: rand(*s, seed=width + i).to(dtype)
    table, a, b, c, wa, wb, w1, step = r(0, V, width), 3.0 * r(1, T, width), 0.1 * r(2, T, width), r(3, T, width), r(4, width), r(5, width), r(6, width), r(7, width)
    ids = torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(0))
    D = lambda t: t.to(device)
    x, n1 = torch.empty(T, width, device=device), torch.empty(T, width, dtype=dtype, device=device)
    residual_norm(x, ids=D(ids), table=D(table), step=D(step), w1=D(w1), n1=n1, eps=1e-4)
    d = lambda t: t.double()
    h = d(table)[ids] + d(step)
    assert rel(x, h) < 1e-6 and rel(n1, oracle.rms(h, d(w1), 1e-4)) < TOL[dtype]
    mix = dict(a=D(a), b=D(b), norm_a=D(wa), norm_b=D(wb), ab_scale=0.5, mult=0.3)
    h1 = h + 0.3 * (0.5 * (oracle.rms(d(a), d(wa), 1e-4) + oracle.rms(d(b), d(wb), 1e-4)) + d(c))
    residual_norm(x, c=D(c), ids=D(ids), inject=D(table), step=D(step), w1=D(w1), n1=n1, eps=1e-4, **mix)
    h1 = h1 + d(table)[ids] + d(step)
    assert rel(x, h1) < 1e-6 and rel(n1, oracle.rms(h1, d(w1), 1e-4)) < TOL[dtype]
    rows, out = i32(6, 0, 6), torch.empty(3, width, dtype=dtype, device=device)
    residual_norm(x, rows=rows.to(device), w1=D(w1), n1=out, store_x=False, eps=1e-4, **mix)
    h2 = h1 + 0.15 * (oracle.rms(d(a), d(wa), 1e-4) + oracle.rms(d(b), d(wb), 1e-4))
    assert rel(x, h1) < 1e-6 and rel(out, oracle.rms(h2[rows.long()], d(w1), 1e-4)) < TOL[dtype]


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda:0", marks=pytest.mark.gpu)])
def test_softcap(device):
    z = torch.linspace(-90.0, 90.0, 1003)
    assert rel(ops.softcap(z.clone().to(device), 7.0), oracle.softcap(z.double(), 7.0)) < 1e-6


# ---------------------------------------------------------------------------------- windowed attention
def attend(q, rows_k, rows_v, cuts, H, KH, hd, scale, window, device, dtype, sink=True, page=64, seed=0):
    """``q`` [T, H, hd] over keys and values [T, KH, hd] in shuffled pages; the queries in portions of the sizes ``cuts``."""
    T = q.shape[0]
    bt, pages, slots = paged(T, page, seed)
    kv = torch.full((pages, 2, 2, KH, page, hd), 3.0)
    for i, rows in ((0, rows_k), (1, rows_v)):
        kv[slots // page, i, 1, :, slots % page] = rows.float()
    kv, bt = kv.to(device, dtype), bt.to(device)
    sinks, out, at = torch.zeros(H, device=device) if sink is True else sink, [], 0
    for n in cuts:
        ql = i32(n).to(device)
        plan = tensor_core_plan(H // KH, hd, dtype, page, i32(0).to(device), ql, n, n == 1)
        out.append(window_attention(q[at: at + n].reshape(n, -1).to(device, dtype), kv, 1, bt, i32(0).to(device), ql, i32(at + n).to(device),
                                    H, KH, scale, window or 0, sinks, plan))
        at += n
    return torch.cat(out).view(T, H, hd)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,KH,hd", [(4, 1, 128), (4, 4, 64), (32, 2, 128), (16, 2, 64), (2, 1, 136), (51, 3, 128), (8, 1, 128)])
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 100, None])
def test_window_attention(H, KH, hd, window, device, dtype):
    """Whole prompts, portions down to two tokens, and decoding, windows around the page size."""
    T = 200
    q, k, v = (rand(T, h, hd, seed=i).to(dtype).double() for i, h in enumerate((H, KH, KH)))
    want = oracle.window_attention(q, k, v, 0.3, window)
    for cuts in ((T,), (63, 2, 1, 64, 1, 1, 68), (130, 70)):
        got = attend(q, k, v, cuts, H, KH, hd, 0.3, window, device, dtype)
        assert rel(got, want) < TOL[dtype], cuts


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,KH,hd", [(4, 1, 128), (2, 2, 64)])
@pytest.mark.parametrize("window", [5, 64, 90])
def test_one_key_at_the_edge_of_the_window(H, KH, hd, window, device, dtype):
    """One key stands out for every query: the query ``window - 1`` places after it finds it, the next one does not, and no
    query finds it before its place; at either side of page borders, from prompts and from decoding."""
    T = 230
    for place in (0, 1, 62, 63, 64, 65, 127, 128):
        q, k, v = (0.1 * rand(T, h, hd, seed=place + i) for i, h in enumerate((H, KH, KH)))
        q[:, :, 3] = 4.0
        k[place, :, 3] = 4.0
        v[place, :, 5] = 20.0
        q, k, v = (t.to(dtype).double() for t in (q, k, v))
        want = oracle.window_attention(q, k, v, 1.0, window)
        last = place + window - 1
        assert want[place: last + 1, :, 5].min() > 15
        assert want[last + 1:, :, 5].abs().max() < 1 and (place == 0 or want[:place, :, 5].abs().max() < 1)
        for cuts in ((T,), (last, 1, 1, T - last - 2), (place + 1, T - place - 1)):
            got = attend(q, k, v, [n for n in cuts if n > 0], H, KH, hd, 1.0, window, device, dtype)
            assert rel(got, want) < TOL[dtype], (place, cuts)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("level", [-150.0, -8.0, 0.0, 9.0, 150.0])
def test_zero_sink(level, device, dtype):
    """Scores far below the sink leave nothing of the values, scores far above leave no trace of the sink."""
    T, H, KH, hd, window = 150, 4, 2, 128, 70
    q, k, v = (rand(T, h, hd, seed=i) for i, h in enumerate((H, KH, KH)))
    q, k = 0.05 * q, 0.05 * k
    q[..., 0] = 10.0
    k[..., 0] = level / 10.0
    q, k, v = (t.to(dtype).double() for t in (q, k, v))
    want = oracle.window_attention(q, k, v, 1.0, window)
    for cuts in ((T,), (T - 2, 1, 1)):
        got = attend(q, k, v, cuts, H, KH, hd, 1.0, window, device, dtype)
        if want.abs().max() > 1e-30:
            assert rel(got, want) < TOL[dtype]
        else:
            assert got.float().abs().max() < 1e-30


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("sink", [None, -4.0, 3.0])
def test_window_without_or_with_another_sink(sink, device, dtype):
    """The kernels take any sink score per head, or none; scores far from zero on both sides of the window's edge."""
    T, H, KH, hd, window = 260, 4, 1, 128, 100
    q, k, v = (rand(T, h, hd, seed=i) for i, h in enumerate((H, KH, KH)))
    q[..., 0], k[..., 0] = 12.0, -12.0
    q, k, v = (t.to(dtype).double() for t in (q, k, v))
    i, j = torch.arange(T).view(T, 1), torch.arange(T).view(1, T)
    s = torch.einsum("thd,jd->htj", q, k[:, 0]).masked_fill((j > i) | (i - j >= window), float("-inf"))
    sinks = None if sink is None else sink - 140.0 + torch.arange(H).double()
    if sinks is not None:
        s = torch.cat([s, sinks.view(H, 1, 1).expand(H, T, 1)], -1)
    want = torch.einsum("htj,jd->thd", torch.softmax(s, -1)[..., :T], v[:, 0])
    for cuts in ((T,), (T - 2, 1, 1)):
        got = attend(q, k, v, cuts, H, KH, hd, 1.0, window, device, dtype, sink=None if sinks is None else sinks.float().to(device))
        assert rel(got, want) < TOL[dtype]


@pytest.mark.gpu
@pytest.mark.parametrize("H,KH,hd", [(8, 2, 128), (8, 8, 64), (16, 1, 128), (3, 3, 128)])
@pytest.mark.parametrize("decode", [True, False])
@pytest.mark.parametrize("window", [70, 256, 0])
def test_tensor_core_attention_agrees(H, KH, hd, decode, window):
    """Ragged batches on the tensor-core kernels (decoding split over the keys or not) against the CUDA-core kernel."""
    for lens in ([700, 1, 64, 65, 333], [129 + 7 * i for i in range(90)]):
        qn = [1] * len(lens) if decode else [min(n, 1 + 61 * i % 150) for i, n in enumerate(lens)]
        B, page, T = len(lens), 64, sum(qn)
        need = [-(-n // page) for n in lens]
        bt = torch.zeros(B, max(need), dtype=torch.int32)
        perm = torch.randperm(sum(need), generator=torch.Generator().manual_seed(1)).int()
        for b, n in enumerate(need):
            bt[b, :n] = perm[sum(need[:b]): sum(need[:b]) + n]
        kv, q = rand(sum(need), 2, 2, KH, page, hd, seed=2).bfloat16().cuda(), rand(T, H * hd, seed=3).bfloat16().cuda()
        ql, kl, bt = i32(*qn).cuda(), i32(*lens).cuda(), bt.cuda()
        qs, sink = (torch.cumsum(ql, 0) - ql).int(), rand(H, seed=4).cuda()
        args = (1, bt, qs, ql, kl, H, KH, hd ** -0.5, window, sink)
        got = window_attention(q, kv, *args, tensor_core_plan(H // KH, hd, torch.bfloat16, page, qs, ql, T, decode))
        want = window_attention(q.float(), kv.float(), *args, None)
        assert rel(got, want.cpu()) < 1e-2
    ops.check_device_error()


# ---------------------------------------------------------------------------------- lightning attention
def lightning_mixer(b, t, W, device, dtype, eps=1e-5):
    c = LightningConfig(b["heads"], b["dim"], b["vdim"], tuple(b["decay"]), eps)
    tensors = {k.split("right.")[1]: v for k, v in t.items() if k.startswith("l0.mix.right.")}
    m = LightningAttention(c, tensors, W, device, dtype)
    w_in = m.w_in.to(device, dtype)

    def run(x, state, idx, qs, ql, kl, one):
        px = ops.linear(x, w_in)
        px[:, : m.act_rows] = oracle.silu(px[:, : m.act_rows].float()).to(dtype)
        return ops.linear(m(px, state, idx, qs, ql, kl, one), m.w_o)

    return c, run


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,d,dv,decay", [(3, 20, 28, None), (1, 128, 128, [0.999]), (2, 64, 96, [1.0, 0.02]), (4, 96, 64, [0.9, 0.5, 0.99, 0.3]),
                                          (2, 40, 200, [0.7, 0.95]), (1, 9, 7, [0.0]), (2, 136, 24, [0.9, 0.99]), (1, 300, 16, [0.97])])
def test_lightning_mixer(H, d, dv, decay, device, dtype):
    """Two sequences in portions beside each other (one of them decoding) against the token-by-token equations; the state
    lives in slots that held something else before."""
    W = 104
    cfg = config(layer(rheads=H, rdim=d, rvdim=dv, decay=decay), width=W)
    t, b = weights_for(cfg, seed=H), cfg["layers"][0]["mixer"]["right"]
    c, run = lightning_mixer(b, t, W, device, dtype)
    w = {k: v.double() for k, v in t.items()}
    h = {s: rand(n, W, seed=n).to(dtype).double() for s, n in (("a", 275), ("b", 140))}
    want = {s: oracle.right_mixer(x, w, "l0.mix.right.", b, 1e-5) for s, x in h.items()}
    state = torch.full((5, *c.state_shapes()["lightning"]), 3.0, device=device)
    at, got, slot = {"a": 0, "b": 0}, {"a": [], "b": []}, {"a": 3, "b": 1}
    for step in ([("a", 2)], [("a", 1), ("b", 64)], [("b", 2), ("a", 131)], [("a", 1), ("b", 1)], [("b", 63), ("a", 2)], [("a", 1)], [("a", 1)],
                 [("a", 65), ("b", 10)], [("a", 71)]):
        x = torch.cat([h[s][at[s]: at[s] + n] for s, n in step]).to(device, dtype)
        ql = i32(*[n for _, n in step])
        kl = i32(*[at[s] + n for s, n in step])
        qs = (torch.cumsum(ql, 0) - ql).int()
        y = run(x, state, i32(*[slot[s] for s, _ in step]).to(device), qs.to(device), ql.to(device), kl.to(device), all(n == 1 for _, n in step))
        for (s, n), o in zip(step, qs.tolist()):
            got[s].append(y[o: o + n, :W])
            at[s] += n
    for s in h:
        assert at[s] == h[s].shape[0]
        assert rel(torch.cat(got[s]), want[s]) < TOL[dtype], s
    assert (state[[0, 2, 4]] == 3.0).all()                           # nobody else's slot was written
    # the state itself: fp32, exact up to rounding of its inputs
    k = oracle.silu(h["a"] @ w["l0.mix.right.k"].T).view(-1, H, d)
    v = oracle.silu(h["a"] @ w["l0.mix.right.v"].T).view(-1, H, dv)
    _, S = oracle.decayed_sum(k, k, v, torch.tensor(b["decay"], dtype=torch.float64))
    assert state.dtype == torch.float32 and rel(state[3, :, :dv, :d], S.transpose(1, 2)) < TOL[dtype]
    assert (state[3, :, dv:] == 0).all() and (state[3, :, :, d:] == 0).all()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("gap", [1, 63, 64, 65, 128, 190])
def test_lightning_remembers_one_token(gap, device, dtype):
    """One key and value stand out; ``gap`` tokens later the state holds decay^gap of it, across the chunks of a prompt and
    across portions."""
    W, H, d = 104, 2, 32
    b = dict(heads=H, dim=d, vdim=d, decay=[0.99, 0.9])
    c = LightningConfig(H, d, d, (0.99, 0.9), 1e-5)
    m = LightningAttention(c, {"q": torch.zeros(H * d, W), "k": torch.zeros(H * d, W), "v": torch.zeros(H * d, W), "g": torch.zeros(H * d, W),
                               "norm": torch.ones(H * d), "o": torch.zeros(W, H * d)}, W, device, dtype)
    T, place = 200, 5
    q, k, v = torch.ones(T, H, d), torch.zeros(T, H, d), torch.zeros(T, H, d)
    k[place], v[place] = 1.0, 2.0
    x = torch.cat([t.reshape(T, -1) for t in (q, k, v)], 1).to(device, dtype)
    want, _ = oracle.decayed_sum(q.double(), k.double(), v.double(), torch.tensor(b["decay"], dtype=torch.float64))
    assert want[place + gap, 0, 0] == pytest.approx(64 * 0.99 ** gap)
    from modular_b200._native import lib

    for cuts in ((T,), (place + gap, T - place - gap)):
        state, at, outs = torch.full((1, *c.state_shapes()["lightning"]), -1.0, device=device), 0, []
        for n in cuts:
            xs, o = x[at: at + n].contiguous(), torch.empty(n, H * d, dtype=dtype, device=device)
            args = (state, i32(0).to(device), i32(0).to(device), i32(n).to(device), i32(at + n).to(device))
            if device == "cpu":
                m.scan_reference(xs, o, *args)
            else:
                lib().lightning(xs, 0, m.k_off, m.v_off, m.decay, m.decay_pow, o, *args, H, d, d, n == 1)
            outs.append(o)
            at += n
        got = torch.cat(outs).view(T, H, d)
        assert (got[:place] == 0).all()
        assert rel(got[place + gap], want[place + gap]) < (1e-5 if dtype == torch.float32 else 4e-3)


@pytest.mark.gpu
@pytest.mark.parametrize("H,d,dv", [(3, 128, 128), (2, 24, 40), (1, 96, 64), (5, 64, 72), (2, 32, 8)])
def test_lightning_chunks_agree_with_the_scan(H, d, dv):
    """The tensor-core kernel on bf16 activations against the fp32 scan of the same values: outputs up to their rounding, the
    state far closer than 16 bits would allow."""
    from modular_b200._native import lib

    lens, gone = [1, 2, 63, 64, 65, 200, 129], [0, 5, 0, 70, 1, 0, 64]
    T, B, dp = sum(lens), len(lens), lib().delta_dim_pad(d)
    decay = torch.tensor([0.999, 0.6, 0.97, 1.0, 0.05])[:H]
    powers = (decay.double().unsqueeze(1) ** torch.arange(65)).float().cuda()
    x = rand(T, H * (2 * d + dv), seed=H).bfloat16().cuda()
    ql, kl = i32(*lens).cuda(), i32(*[n + g for n, g in zip(lens, gone)]).cuda()
    qs, idx, init = (torch.cumsum(ql, 0) - ql).int(), i32(3, 0, 6, 2, -1, 1, 5).cuda(), rand(8, H, dv, dp, seed=1).cuda()
    init[..., d:] = 0
    got = []
    for dtype in (torch.bfloat16, torch.float32):
        st, o = init.clone(), torch.zeros(T, H * dv, dtype=dtype, device="cuda")
        lib().lightning(x.to(dtype), 0, H * d, 2 * H * d, decay.cuda(), powers, o, st, idx, qs, ql, kl, H, d, dv, False)
        got.append((o, st))
    assert rel(got[0][1], got[1][1].cpu()) < 2e-5 and rel(got[0][0], got[1][0].cpu()) < 3e-3
    assert torch.equal(got[0][1][[4, 7]], init[[4, 7]])


@pytest.mark.parametrize("device,dtype", RUNS)
def test_lightning_without_a_slot(device, dtype):
    """Sequences with slot -1 start from zero and keep nothing (the dummies of a padded decode batch)."""
    W = 104
    cfg = config(layer(), width=W)
    t, b = weights_for(cfg), cfg["layers"][0]["mixer"]["right"]
    c, run = lightning_mixer(b, t, W, device, dtype)
    state = torch.ones((2, *c.state_shapes()["lightning"]), device=device)
    dev = lambda *v: i32(*v).to(device)
    w = {k: v.double() for k, v in t.items()}
    for lens in ((1, 1), (70, 3)):
        x = rand(sum(lens), W).to(device, dtype)
        y = run(x, state, dev(-1, -1), dev(0, lens[0]), dev(*lens), dev(lens[0], 99), lens == (1, 1))
        for lo, hi in ((0, lens[0]), (lens[0], sum(lens))):
            assert rel(y[lo: hi, :W], oracle.right_mixer(x[lo: hi].cpu().double(), w, "l0.mix.right.", b, 1e-5)) < TOL[dtype]
    assert (state == 1).all()


# ---------------------------------------------------------------------------------- one block
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("l", [layer(), layer(heads=1, kv_heads=1, dim=8, vdim=8, dims=2, window=3, rheads=1, rdim=8, rvdim=8, ff=8),
                               layer(heads=5, kv_heads=1, dim=72, vdim=128, dims=72, scaling=YARN, rheads=2, rdim=128, rvdim=72, ff=None),
                               layer(heads=6, kv_heads=3, dim=160, vdim=40, dims=100, window=80, rheads=2, rdim=64, rvdim=64),
                               layer(heads=34, kv_heads=2, dim=16, vdim=32, dims=8, window=1)], ids=["odd", "small", "no ff", "wide head", "many heads"])
def test_parallel_block(l, device, dtype):
    """Both mixers and the feed-forward of one layer over a prompt in two portions and two decoded tokens."""
    W, T, page = 104, 150, 64
    cfg = config(l, width=W)
    t, c = weights_for(cfg, seed=1), VipotarConfig.from_hf(cfg)
    side = lambda s: {n.rsplit(".", 1)[1]: v for n, v in t.items() if n.startswith(f"l0.mix.{s}.")}
    left, hd = c.attention(0), c.head_width
    block = ParallelBlock(WindowAttention(left, side("left"), hd, W, device, dtype), LightningAttention(c.lightning(0), side("right"), W, device, dtype),
                          t["l0.mix.left.out"], t["l0.mix.right.out"], t.get("l0.mlp.up"), t.get("l0.mlp.down"), W, device, dtype)
    h, w = rand(T, W, seed=2).to(dtype), {k: v.double() for k, v in t.items()}
    want = oracle.parallel_mixer(h.double(), w, "l0.mix.", l["mixer"], 1e-5)
    if l["mlp"]:
        want = want + oracle.dense_ff(h.double(), w, "l0.mlp.")
    bt, pages, slots = paged(T, page)
    kv = torch.zeros(pages, 2, 1, left.kv_heads, page, hd, dtype=dtype, device=device)
    state = torch.ones((1, *c.lightning(0).state_shapes()["lightning"]), device=device)
    cs = cos_sin_table(left.rot_dims, T, left.rope_base, left.rope_scaling, device)
    D = lambda *v: i32(*v).to(device)
    got, at = torch.zeros(T, W, device=device), 0
    for n in (85, 63, 1, 1):
        plan = tensor_core_plan(left.group_pad, hd, dtype, page, D(0), D(n), n, n == 1)
        out = block(h[at: at + n].to(device), ops.linear, kv, 0, state, cs, torch.arange(at, at + n, dtype=torch.int32, device=device),
                    slots[at: at + n].to(device), bt.to(device), D(0), D(n), D(at + n), D(0), plan, n == 1)
        residual_norm(got[at: at + n], eps=1e-5, cols=W, **out)
        at += n
    assert rel(got, want) < TOL[dtype]


# ---------------------------------------------------------------------------------- whole models
MIXED = config(layer(scaling=YARN), layer(heads=4, kv_heads=4, dim=24, vdim=56, window=64, dims=24, rheads=2, rdim=40, rvdim=16, ff=None),
               layer(heads=3, kv_heads=1, dim=64, vdim=64, window=100, dims=8, rheads=5, rdim=8, rvdim=24, ff=200),
               layer(heads=2, kv_heads=2, dim=16, vdim=16, window=2, dims=4, rheads=1, rdim=72, rvdim=72),
               loop={"start": 1, "stop": 3, "times": 2})


@pytest.fixture(scope="module")
def mixed_model():
    t = weights_for(MIXED)
    draw = lambda n, s: torch.randint(0, MIXED["vocab"], (n,), generator=torch.Generator().manual_seed(s)).tolist()
    return t, {r: (toks, oracle.forward(MIXED, t, toks)) for r, toks in (("a", draw(300, 3)), ("b", draw(150, 4)))}


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
def test_residual_stream_of_every_run(mixed_model, device, dtype):
    t, ref = mixed_model
    toks, (_, want) = ref["b"]
    llm = engine(MIXED, t, device, dtype)
    ctx = TextContext.from_prompt(toks, llm.max_length, "r")
    llm.kv.claim(ctx)
    llm.kv.alloc(ctx)
    b = llm.pipeline.packer.step_tensors(llm.pipeline.packer.pack([ctx], llm.kv))
    stream = []
    llm.model._forward(b["tokens"], b["positions"], b["slots"], b["block_table"], b["q_start"], b["q_len"], b["kv_len"],
                       b["logit_rows"], b["state_slot"], stream=stream)
    assert len(stream) == len(want) == 6 and stream[0].dtype == torch.float32
    for i, (got, exp) in enumerate(zip(stream, want)):
        assert rel(got, exp) < TOL[dtype], f"after run {i}"


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
    t, ref = mixed_model
    out = replay(engine(MIXED, t, device, dtype), {r: v[0] for r, v in ref.items()}, SCHEDULES[name])
    for r, got in out.items():
        want = ref[r.split("#")[0]][1][0]
        err = (got.double() - want).pow(2).mean(1).sqrt() / want.pow(2).mean().sqrt()
        assert err.max() < 2 * TOL[dtype], (r, int(err.argmax()))


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("cfg", [
    config(layer()), config(layer(heads=1, kv_heads=1, dim=4, vdim=4, dims=2, window=1, rheads=1, rdim=4, rvdim=4, ff=4), width=40, vocab=33),
    config(layer(), layer(window=9), loop={"start": 0, "stop": 2, "times": 3}, mult=1.0, cap=40.0),
    config(layer(), layer(dim=64, vdim=128, dims=64, scaling=YARN), layer(ff=None), loop={"start": 2, "stop": 3, "times": 1}, eps=1e-3, width=136, vocab=258),
    config(layer(heads=10, kv_heads=2, dim=104, vdim=80, dims=60, rheads=7, rdim=104, rvdim=48, ff=264), layer(), width=200, vocab=98,
           loop={"start": 0, "stop": 1, "times": 2}),
    config(layer(dim=200, vdim=144, dims=66, window=70, rheads=2, rdim=144, rvdim=8), width=88)],
    ids=["no loop", "tiny", "all looped", "last looped", "wide", "wide heads"])
def test_other_sizes(cfg, device, dtype):
    t = weights_for(cfg, seed=11)
    toks = torch.randint(0, cfg["vocab"], (170,), generator=torch.Generator().manual_seed(1)).tolist()
    want = oracle.forward(cfg, t, toks)[0]
    out = replay(engine(cfg, t, device, dtype), {"a": toks}, [[("a", n)] for n in (40, 2, 1, 1, 21, 1, 104)])
    assert rel(out["a"], want) < TOL[dtype]


@pytest.mark.parametrize("device,dtype", [RUNS[0], RUNS[2]])
def test_pages_of_other_sizes(device, dtype):
    """Pages that are a multiple of 64 tokens and pages that are not (no tensor-core attention then)."""
    cfg = config(layer(window=50), layer(window=150))
    t = weights_for(cfg, seed=12)
    toks = torch.randint(0, cfg["vocab"], (260,), generator=torch.Generator().manual_seed(1)).tolist()
    want = oracle.forward(cfg, t, toks)[0]
    for page in (128, 40):
        out = replay(engine(cfg, t, device, dtype, page=page), {"a": toks}, [[("a", n)] for n in (129, 1, 1, 60, 69)])
        assert rel(out["a"], want) < TOL[dtype], page


@pytest.mark.parametrize("device,dtype", RUNS)
def test_greedy_generation(device, dtype):
    """More requests than a batch holds through the scheduler, prompts in chunks beside decoding, with preemption when the
    pool runs dry: the tokens are those of plain greedy decoding."""
    cfg = config(layer(window=30), layer(heads=2, kv_heads=1, ff=None), vocab=150, cap=20.0, loop={"start": 0, "stop": 1, "times": 2})
    t = weights_for(cfg, seed=21)
    t["head"] = t["head"] * 4.0                                    # clear winners
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
        top = want.max(-1).values
        chosen = want[torch.arange(24), r.tokens]
        assert (top - chosen).max() < (1e-3 if dtype == torch.float32 else 0.5)      # never worse than a near tie
        exact += int((want.argmax(-1) == torch.tensor(r.tokens)).sum())
        total += 24
    assert exact >= total * (1.0 if dtype == torch.float32 else 0.9)
    assert llm.kv.free_state_slots == 3 and llm.kv.used_blocks_pct == 0 and llm.kv.preemptions > 0
    if device != "cpu":
        assert llm.model.graph_replays > 0


@pytest.mark.gpu
def test_sampling_and_penalties_on_gpu():
    cfg = config(layer(), layer())
    llm = engine(cfg, weights_for(cfg), "cuda:0", torch.bfloat16, max_logit_rows=0)
    sp = lambda seed: SamplingParams(temperature=1.0, top_k=20, max_new_tokens=16, ignore_eos=True, seed=seed, repetition_penalty=1.2)
    a, b = (llm.generate([[1, 2, 3], [4, 5]], [sp(s), sp(s + 1)]) for s in (5, 9))
    assert all(len(r.tokens) == 16 and 0 <= min(r.tokens) and max(r.tokens) < cfg["vocab"] for r in a + b)
    assert [r.tokens for r in a] != [r.tokens for r in b]


# ---------------------------------------------------------------------------------- configuration, command line
def test_config_checks_and_registry():
    arch = PIPELINE_REGISTRY.retrieve_architecture(MIXED)
    assert arch.name == "Vipotar" and arch.config_class is VipotarConfig
    c = VipotarConfig.from_hf(MIXED)
    again = VipotarConfig.from_hf(c.to_hf())
    assert again.layers == c.layers and again.runs == c.runs and PIPELINE_REGISTRY.retrieve_architecture(c.to_hf()) is arch
    assert [(r.layer, r.step, r.inject) for r in c.runs] == [(0, -1, False), (1, 0, False), (2, -1, False), (1, 1, True), (2, -1, False), (3, -1, False)]
    assert c.head_width == 64 and c.cache_heads == 4 and len(c.state_specs()) == 6
    assert head_width(65) == 128 and head_width(130) == 136
    t = weights_for(MIXED)
    assert {n: tuple(v.shape) for n, v in t.items()} == c.tensor_shapes()
    for bad in (config(layer(heads=5, kv_heads=2)), config(layer(decay=[0.5])), config(layer(dims=50)),
                config(layer(), loop={"start": 0, "stop": 2, "times": 2}), config(layer(), loop={"start": 0, "stop": 1, "times": 0})):
        with pytest.raises(ValueError):
            VipotarConfig.from_hf(bad)
    with pytest.raises(KeyError):
        VipotarWeights.from_state_dict(c, {k: v for k, v in t.items() if k != "l2.mix.right.norm"}, "cpu", torch.float32)
    with pytest.raises(ValueError):
        VipotarWeights.from_state_dict(c, {**t, "l2.mix.left.q": t["l2.mix.left.q"][:-1]}, "cpu", torch.float32)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_trace_replay_program(tmp_path, device, dtype):
    """The command-line replay: a checkpoint folder in, steps on standard input, logits in files."""
    cfg = config(layer(window=20), layer(), loop={"start": 1, "stop": 2, "times": 2})
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
    assert rel(load(0), want["a"][[0, 3]]) < TOL[dtype]
    assert rel(load(2), torch.stack([want["a"][5], want["b"][69], want["b"][67]])) < TOL[dtype]
    assert rel(load(3), want["a"][5:6]) < TOL[dtype]
