"""Gotunex against the plain implementation in ``gotunex_oracle``: every mechanism alone, then whole models through the
engine's own step (portions, mixed batches, reused pages and slots, far keys, long decoding) and greedy generation through
its scheduler. CPU runs take the package's PyTorch operations in fp32; GPU runs take the kernels in fp32 and bf16."""

import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import gotunex_oracle as oracle  # noqa: E402
from modular_b200.entrypoints.llm import LLM
from modular_b200.entrypoints.trace import TraceSession
from modular_b200.kv_cache import InsufficientBlocksError, KVCacheParams, PagedKVCacheManager
from modular_b200.models.gotunex import GotunexConfig, GotunexWeights
from modular_b200.nn.delta_rule import DeltaRule, DeltaRuleConfig, dim_pad
from modular_b200.nn.latent_attention import LatentAttention, LatentAttentionConfig, latent_attention
from modular_b200.nn.moe import TableRouter, expert_mlp
from modular_b200.nn.residual import residual_norm
from modular_b200.nn.rotary_embedding import cos_sin_table
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


def latent(heads=4, dim=40, rot_dim=24, vdim=56, kv_rank=72, q_rank=48, base=5000.0, **kw):
    return {"type": "latent_attention", "mixer": dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank,
                                                      scale=0.9 * (dim + rot_dim) ** -0.5, rot=dict(base=base, dims=rot_dim), **kw)}


def delta(heads=6, kv_heads=3, dim=24, vdim=40, conv=4):
    return {"type": "channel_delta", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)}


def dense(ff=136):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=72):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(*layers, width=120, vocab=190, eps=1e-5, scale=3.0):
    """``layers``: (mixer entry, feed-forward entry or None)."""
    return {"architecture": "Gotunex", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "layers": [{**copy.deepcopy(m), "mlp": ff} for m, ff in layers]}


def weights_for(cfg, seed=0, decay_rank=20, gate_rank=28, dtype=torch.bfloat16):
    """Random tensors of a checkpoint, rounded to ``dtype``."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    lin = lambda o, i: rnd(o, i) * i ** -0.5
    norm = lambda n: 1.0 + 0.2 * rnd(n)
    W, V = cfg["width"], cfg["vocab"]
    t = {"embed": rnd(V, W), "final.norm": norm(W), "head": lin(V, W)}
    for i, l in enumerate(cfg["layers"]):
        m, p, ff = l["mixer"], f"l{i}.mix.", l["mlp"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        t[f"l{i}.norm1"] = norm(W)
        if l["type"] == "latent_attention":
            r, R, Q = m["rot_dim"], m["kv_rank"], m["q_rank"]
            t.update({p + "dq": lin(Q, W), p + "dq.norm": norm(Q), p + "uq": 2.0 * lin(H * (d + r), Q), p + "uk": lin(H * d, R),
                      p + "uv": lin(H * dv, R), p + "sink": rnd(H), p + "g": lin(H * dv, W), p + "o": lin(W, H * dv)})
            if "kv_from" not in m:
                t.update({p + "dkv": lin(R + r, W), p + "dkv.norm": norm(R)})
        else:
            K = m["kv_heads"] * d
            for n, rows in (("q", K), ("k", K), ("v", H * dv)):
                t[p + n], t[p + n + ".conv"] = lin(rows, W), rnd(rows, m["conv"]) * m["conv"] ** -0.5
            t.update({p + "b": lin(H, W), p + "A_log": rnd(H) * 0.5 - 1.0, p + "norm": norm(dv), p + "a1": lin(decay_rank, W),
                      p + "a2": lin(H * d, decay_rank), p + "dt_bias": rnd(H * d) - 2.0, p + "g1": lin(gate_rank, W),
                      p + "g2": lin(H * dv, gate_rank), p + "o": lin(W, H * dv)})
        if ff is not None:
            t[f"l{i}.norm2"] = norm(W)
            if ff["kind"] == "dense":
                t.update({f"l{i}.mlp.up": lin(ff["ff"], W), f"l{i}.mlp.down": lin(W, ff["ff"])})
            else:
                for e in range(ff["router"]["experts"]):
                    t.update({f"l{i}.mlp.e{e}.{n}": lin(*s) for n, s in (("gate", (ff["expert"]["ff"], W)), ("up", (ff["expert"]["ff"], W)),
                                                                          ("down", (W, ff["expert"]["ff"])))})
                t[f"l{i}.mlp.table"] = torch.stack([torch.randperm(ff["router"]["experts"], generator=g)[: ff["router"]["top"]]
                                                    for _ in range(V)]).int()
    return {k: v if v.dtype == torch.int32 else v.to(dtype).float() for k, v in t.items()}


def engine(cfg, t, device, dtype, tokens=512, page=64, batch=4, **kw):
    c = GotunexConfig.from_hf(cfg)
    args = dict(max_length=tokens, max_batch_size=batch, max_batch_input_tokens=tokens, page_size=page,
                num_kv_pages=-(-tokens // page) + 1, enable_prefix_caching=False, max_logit_rows=tokens,
                enable_overlap_scheduler=False, graph_batch_sizes=[1, 4])
    args.update(kw)
    return LLM(c, GotunexWeights.from_state_dict(c, t, device, dtype), device=device, dtype=dtype, **args)


MIXED = config((latent(), dense()), (delta(), moe()), (latent(heads=3, dim=24, vdim=24, q_rank=64, kv_rank=136, rot_dim=16, base=700.0), moe(top=1)),
               (latent(heads=5, dim=72, vdim=16, q_rank=40, kv_from=0), None), (delta(heads=3, kv_heads=1, dim=72, vdim=20, conv=2), dense(200)),
               (latent(heads=2, dim=16, vdim=48, kv_rank=136, rot_dim=16, base=700.0, kv_from=2), moe(experts=7, top=3)))


@pytest.fixture(scope="module")
def mixed_model():
    t = weights_for(MIXED)
    toks = torch.randint(0, MIXED["vocab"], (300,), generator=torch.Generator().manual_seed(3)).tolist()
    other = torch.randint(0, MIXED["vocab"], (150,), generator=torch.Generator().manual_seed(4)).tolist()
    return t, {"a": (toks, oracle.forward(MIXED, t, toks)), "b": (other, oracle.forward(MIXED, t, other))}


# ---------------------------------------------------------------------------------- mechanisms alone
def paged(n_tokens, page, seed=0):
    """A block table of shuffled pages for one sequence: (table [1, n], pages in the pool, slots of every position)."""
    n = -(-n_tokens // page)
    pages = torch.randperm(n + 2, generator=torch.Generator().manual_seed(seed))[:n].int()
    pos = torch.arange(n_tokens)
    return pages.view(1, -1), n + 2, pages.long()[pos // page] * page + pos % page


def i32(*v):
    return torch.tensor(v, dtype=torch.int32)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("m", [latent(), latent(heads=1, dim=8, rot_dim=8, vdim=8, kv_rank=16, q_rank=8),
                               latent(heads=7, dim=130, rot_dim=64, vdim=100, kv_rank=300, q_rank=200),
                               latent(heads=2, dim=32, rot_dim=72, vdim=32, kv_rank=64, q_rank=96),
                               latent(heads=16, dim=64, rot_dim=32, vdim=64, kv_rank=520, q_rank=64)],
                         ids=["odd", "small", "wide", "rot72", "latent520"])
def test_latent_attention_mixer(m, device, dtype):
    """One mixer over a prompt in two portions and two decoded tokens, pages in shuffled order."""
    cfg = config((m, None), width=104)
    t, m = weights_for(cfg, seed=1), m["mixer"]
    c = LatentAttentionConfig(m["heads"], m["dim"], m["rot_dim"], m["rot"]["dims"], m["vdim"], m["kv_rank"], m["q_rank"], m["scale"],
                              m["rot"]["base"], 1e-5)
    mix = LatentAttention(c, {k[len("l0.mix."):]: v for k, v in t.items() if k.startswith("l0.mix.")}, 104, device, dtype)
    T, page = 150, 64
    h = torch.randn(T, 104, generator=torch.Generator().manual_seed(2)).to(dtype).double()
    w = {k: v.double() for k, v in t.items() if v.dtype != torch.int32}
    want = oracle.latent_attention(h, w, "l0.mix.", m, 1e-5, oracle.latent_rows(h, w, "l0.mix.", m, 1e-5))
    bt, pages, slots = paged(T, page)
    cache = torch.full((pages, page, c.cache_width + 8), 7.0, dtype=dtype, device=device)
    cs = cos_sin_table(c.rot_dims, T, c.rope_base, None, device)
    from modular_b200 import ops

    got, at = [], 0
    for n in (85, 63, 1, 1):
        x = h[at: at + n].to(device, dtype)
        got.append(mix(x, ops.linear, cache, cs, torch.arange(at, at + n, dtype=torch.int32, device=device), slots[at: at + n].to(device),
                       bt.to(device), i32(0).to(device), i32(n).to(device), i32(at + n).to(device), n == 1))
        at += n
    assert rel(torch.cat(got)[:, :104], want) < TOL[dtype]


@pytest.mark.parametrize("device,dtype", RUNS)
def test_far_keys_at_page_borders(device, dtype):
    """One key stands out for every query: attention must find it at either side of every page border, from prompts and
    from decoding alike, and must not see it before its place."""
    H, Rp, page, T = 3, 128, 64, 200
    gen = torch.Generator().manual_seed(5)
    rows = 0.1 * torch.randn(T, Rp + 64, generator=gen)
    bt, pages, slots = paged(T, page, seed=6)
    mark = torch.zeros(Rp + 64)
    mark[3] = mark[Rp + 2] = 4.0                                   # half of the score from the latent, half from the rotated part
    for place in (0, 1, 62, 63, 64, 65, 127, 128, 191, 192, 198):
        r = rows.clone()
        r[place] += mark
        r = r.to(dtype).float()
        cache = torch.zeros(pages * page, Rp + 64)
        cache[slots] = r
        cache = cache.view(pages, page, -1).to(device, dtype)
        q = (0.1 * torch.randn(T, H, Rp + 64, generator=gen) + mark).to(dtype).float()
        s = torch.einsum("qhd,kd->hqk", q, r).masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
        want = torch.einsum("hqk,kd->qhd", torch.softmax(s, -1), r[:, :Rp])
        assert s[:, place:, place].min() > s[:, place + 1:, :place].max() + 10 if place else True
        for cuts in ((T,), (place or 1, T - (place or 1)), (T - 2, 1, 1)):
            at, got = 0, []
            for n in cuts:
                qq = q[at: at + n].to(device, dtype)
                got.append(latent_attention(qq[..., :Rp].contiguous(), qq[..., Rp:], cache, bt.to(device), i32(0).to(device),
                                            i32(n).to(device), i32(at + n).to(device), 1.0, None, n == 1))
                at += n
            assert rel(torch.cat(got), want) < TOL[dtype], (place, cuts)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("sink", [-60.0, 0.0, 30.0, 200.0])
def test_sink(sink, device, dtype):
    """A sink takes its share of the softmax, once and unscaled: also one far above or below every score."""
    H, Rp, page, T = 5, 64, 64, 90
    g = torch.Generator().manual_seed(7)
    rows, q = torch.randn(T, Rp + 64, generator=g).to(dtype).float(), torch.randn(T, H, Rp + 64, generator=g).to(dtype).float()
    bt, pages, slots = paged(T, page, seed=8)
    cache = torch.zeros(pages * page, Rp + 64)
    cache[slots] = rows
    cache = cache.view(pages, page, -1).to(device, dtype)
    sinks = sink + torch.arange(H).float()
    s = (torch.einsum("qhd,kd->hqk", q, rows) * 0.25).masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf")).double()
    p = torch.softmax(torch.cat([s, sinks.double().view(H, 1, 1).expand(H, T, 1)], -1), -1)[..., :T]
    want = torch.einsum("hqk,kd->qhd", p, rows[:, :Rp].double())
    for lo, hi in ((0, T), (T - 1, T)):
        qq = q[lo: hi].to(device, dtype)
        got = latent_attention(qq[..., :Rp].contiguous(), qq[..., Rp:], cache, bt.to(device), i32(0).to(device), i32(hi - lo).to(device),
                               i32(hi).to(device), 0.25, sinks.to(device), hi - lo == 1)
        if want[lo: hi].abs().max() > 1e-30:
            assert rel(got, want[lo: hi]) < TOL[dtype]
        else:
            assert got.float().abs().max() < 1e-30


@pytest.mark.gpu
@pytest.mark.parametrize("heads,rank", [(128, 512), (12, 512), (6, 192), (96, 384), (67, 64)])
@pytest.mark.parametrize("decode", [True, False])
def test_attention_kernels_agree(heads, rank, decode):
    """The tensor-core kernels (split over the keys or not) against the CUDA-core kernel on the same rows, with sinks."""
    g = torch.Generator(device="cuda").manual_seed(9)
    lens = [700, 1, 64, 65, 333]
    qn = [1] * 5 if decode else [150, 1, 64, 2, 100]
    B, page = len(lens), 64
    need = [-(-n // page) for n in lens]
    bt = torch.zeros(B, max(need), dtype=torch.int32, device="cuda")
    perm = torch.randperm(sum(need), generator=torch.Generator().manual_seed(1)).int().cuda()
    for b, n in enumerate(need):
        bt[b, :n] = perm[sum(need[:b]): sum(need[:b]) + n]
    rows = lambda *s: torch.randn(*s, generator=g, device="cuda", dtype=torch.float32).bfloat16()
    cache, T = rows(sum(need), page, rank + 64), sum(qn)
    q, sink = rows(T, heads, rank + 64), torch.randn(heads, generator=g, device="cuda")
    ql, kl = torch.tensor(qn, dtype=torch.int32, device="cuda"), torch.tensor(lens, dtype=torch.int32, device="cuda")
    qs = (torch.cumsum(ql, 0) - ql).int()
    args = (bt, qs, ql, kl, (rank + 64) ** -0.5, sink, decode)
    got = latent_attention(q[..., :rank].contiguous(), q[..., rank:].contiguous(), cache, *args)
    want = latent_attention(q[..., :rank].float().contiguous(), q[..., rank:].float(), cache.float(), *args)
    assert rel(got, want.cpu()) < 1e-2


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,KH,d,dv,taps", [(4, 4, 32, 32, 4), (6, 2, 24, 40, 3), (3, 1, 72, 9, 2), (2, 2, 128, 128, 4), (2, 1, 100, 136, 1),
                                            (1, 1, 300, 16, 5), (2, 2, 200, 264, 4)])
def test_delta_rule_mixer(H, KH, d, dv, taps, device, dtype):
    """Two sequences in portions beside each other (one of them decoding) against the token-by-token equations; the state
    and the convolution inputs live in slots that held something else before."""
    W = 104
    cfg = config((delta(H, KH, d, dv, taps), None), width=W)
    t, m = weights_for(cfg, seed=H, decay_rank=12, gate_rank=17), cfg["layers"][0]["mixer"]
    c = DeltaRuleConfig(W, H, KH, d, dv, taps, 12, 17, 1e-5)
    mix = DeltaRule(c, {k[len("l0.mix."):]: v for k, v in t.items() if k.startswith("l0.mix.")}, W, device, dtype)
    w = {k: v.double() for k, v in t.items() if v.dtype != torch.int32}
    h = {s: torch.randn(n, W, generator=torch.Generator().manual_seed(n)).to(dtype).double() for s, n in (("a", 75), ("b", 40))}
    want = {s: oracle.channel_delta(x, w, "l0.mix.", m, 1e-5) for s, x in h.items()}
    shapes = c.state_shapes()
    state = torch.full((5, *shapes["delta"]), 3.0, device=device)
    conv = torch.full((5, *shapes["conv"]), -2.0, device=device)
    from modular_b200 import ops

    at, got, slot = {"a": 0, "b": 0}, {"a": [], "b": []}, {"a": 3, "b": 1}
    for step in ([("a", 2)], [("a", 1), ("b", 30)], [("b", 2), ("a", 67)], [("a", 1), ("b", 1)], [("b", 7), ("a", 2)], [("a", 1)], [("a", 1)]):
        x = torch.cat([h[s][at[s]: at[s] + n] for s, n in step]).to(device, dtype)
        ql = i32(*[n for _, n in step])
        kl = i32(*[at[s] + n for s, n in step])
        qs = (torch.cumsum(ql, 0) - ql).int()
        y = mix(x, ops.linear, state, conv, i32(*[slot[s] for s, _ in step]).to(device), qs.to(device), ql.to(device), kl.to(device),
                all(n == 1 for _, n in step))
        for (s, n), o in zip(step, qs.tolist()):
            got[s].append(y[o: o + n, :W])
            at[s] += n
    for s in h:
        assert at[s] == h[s].shape[0] or s == "a"
        assert rel(torch.cat(got[s]), want[s][: at[s]]) < TOL[dtype], s
    assert (state[0] == 3.0).all() and (conv[4] == -2.0).all()       # nobody else's slot was written


@pytest.mark.parametrize("device,dtype", RUNS)
def test_delta_rule_without_a_slot(device, dtype):
    """Sequences with slot -1 start from zero and keep nothing (the dummies of a padded decode batch)."""
    W, d = 104, 32
    cfg = config((delta(2, 2, d, 16, 3), None), width=W)
    t = weights_for(cfg)
    c = DeltaRuleConfig(W, 2, 2, d, 16, 3, 20, 28, 1e-5)
    mix = DeltaRule(c, {k[len("l0.mix."):]: v for k, v in t.items() if k.startswith("l0.mix.")}, W, device, dtype)
    from modular_b200 import ops

    state = torch.ones((2, *c.state_shapes()["delta"]), device=device)
    conv = torch.ones((2, *c.state_shapes()["conv"]), device=device)
    x = torch.randn(2, W, generator=torch.Generator().manual_seed(0)).to(device, dtype)
    dev = lambda *v: i32(*v).to(device)
    y = mix(x, ops.linear, state, conv, dev(-1, -1), dev(0, 1), dev(1, 1), dev(1, 9), True)
    w = {k: v.double() for k, v in t.items() if v.dtype != torch.int32}
    for r in range(2):
        want = oracle.channel_delta(x[r: r + 1].cpu().double(), w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5)
        assert rel(y[r: r + 1, :W], want) < TOL[dtype]
    assert (state == 1).all() and (conv == 1).all()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("experts,top,ff", [(5, 2, 72), (8, 1, 64), (40, 7, 24), (1, 1, 200)])
def test_table_experts(experts, top, ff, device, dtype):
    W, V, T = 96, 50, 77
    cfg = config((delta(), moe(experts, top, ff)), (delta(), moe(3, 3, 16)), width=W, vocab=V)
    t = weights_for(cfg, seed=2)
    g = torch.Generator().manual_seed(1)
    x, toks = torch.randn(T, W, generator=g).to(dtype), torch.randint(0, V, (T,), generator=g)
    router = TableRouter([t["l0.mlp.table"], t["l1.mlp.table"]], [experts, 3], device)
    for i, (inverse, offsets) in enumerate(router.route(toks.to(device))):
        E, k = (experts, top) if i == 0 else (3, 3)
        inv, off = inverse.cpu().long(), offsets.cpu().tolist()
        assert sorted(inv.flatten().tolist()) == list(range(T * k)) and off[0] == 0 and off[-1] == T * k
        expert = t[f"l{i}.mlp.table"][toks].long()
        assert all(off[e] <= p < off[e + 1] for e, p in zip(expert.flatten().tolist(), inv.flatten().tolist()))
        xp = torch.empty(T * k, W, dtype=dtype)
        for j in range(k):
            xp[inv[:, j]] = x
        gu = torch.stack([torch.cat([t[f"l{i}.mlp.e{e}.gate"], t[f"l{i}.mlp.e{e}.up"]]) for e in range(E)]).to(device, dtype)
        dn = torch.stack([t[f"l{i}.mlp.e{e}.down"] for e in range(E)]).to(device, dtype)
        out = expert_mlp(xp.to(device), offsets, gu, dn, T).cpu().double()
        want = oracle.table_moe(x.double(), toks.tolist(), {n: v.double() for n, v in t.items()}, f"l{i}.mlp.", k)
        assert rel(out[inv].sum(1) / k, want) < TOL[dtype]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("width", [64, 200, 1336])
def test_residual_seam(width, device, dtype):
    T, V, k = 9, 30, 3
    g = torch.Generator().manual_seed(width)
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype)
    table, a, b, e, w1, w2 = rnd(V, width), rnd(T, width), rnd(T, width), rnd(T * k, width), rnd(width), rnd(width)
    ids, inv = torch.randint(0, V, (T,), generator=g), torch.randperm(T * k, generator=g).view(T, k).int()
    D = lambda *ts: [x.to(device) for x in ts]
    x = torch.empty(T, width, device=device)
    n1, n2 = torch.empty(T, width, dtype=dtype, device=device), torch.empty(T * k, width, dtype=dtype, device=device)
    dt, da, db, de, dw1, dw2, dids, dinv = D(table, a, b, e, w1, w2, ids, inv)
    residual_norm(x, ids=dids, table=dt, scale=2.5, w1=dw1, n1=n1, w2=dw2, n2=n2, scatter=dinv, eps=1e-4)
    h = table.double()[ids] * 2.5
    assert rel(x, h) < 1e-6 and rel(n1, oracle.rms(h, w1.double(), 1e-4)) < TOL[dtype]
    for j in range(k):
        assert rel(n2[dinv[:, j].long()], oracle.rms(h, w2.double(), 1e-4)) < TOL[dtype]
    residual_norm(x, a=da, b=db)
    h = h + a.double() + b.double()
    assert rel(x, h) < 1e-6
    rows, out = torch.tensor([7, 0, 7], dtype=torch.int32), torch.empty(3, width, dtype=dtype, device=device)
    residual_norm(x, a=da, e=de, inverse=dinv, pair_w=1 / k, rows=rows.to(device), w1=dw1, n1=out, store_x=False, eps=1e-4)
    assert rel(x, h) < 1e-6
    h = h + a.double() + e.double()[inv.long()].mean(1)
    assert rel(out, oracle.rms(h[rows.long()], w1.double(), 1e-4)) < TOL[dtype]


@pytest.mark.parametrize("device,dtype", RUNS)
def test_gelu_and_rotation(device, dtype):
    from modular_b200 import ops
    from modular_b200.nn.latent_attention import rotate_heads

    x = torch.linspace(-9, 9, 400).to(dtype)
    assert rel(ops.gelu_tanh(x.clone().view(4, 100).to(device)), oracle.gelu_tanh(x.double()).view(4, 100)) < TOL[dtype]
    h = torch.randn(3, 4 * 40, generator=torch.Generator().manual_seed(0)).to(dtype)
    y = h.clone().to(device)
    rotate_heads(y, 4, 40, 24, False, i32(5000, 5001, 5002).to(device), cos_sin_table(24, 5003, 300.0, None, device))
    assert rel(y, oracle.rotate(h.double().view(3, 4, 40), 24, 300.0, 5000).view(3, -1)) < TOL[dtype]


@pytest.mark.gpu
@pytest.mark.parametrize("N,K", [(64, 64), (8192, 64), (896, 64), (1280, 72), (2048, 160), (256, 2048), (1408, 64)])
def test_decode_sized_projection(N, K):
    """Projections of few tokens, among them many rows over a single 64-wide block of the inner width."""
    from modular_b200 import ops

    g = torch.Generator().manual_seed(N + K)
    w = torch.randn(N, K, generator=g).bfloat16()
    for M in (1, 5, 64, 256):
        x = torch.randn(M, K, generator=g).bfloat16()
        assert rel(ops.linear(x.cuda(), w.cuda()), x.double() @ w.double().t()) < 1e-2


# ---------------------------------------------------------------------------------- whole models
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
    assert not s.live and llm.kv.used_blocks_pct == 0 and (not llm.kv.state or llm.kv.free_state_slots == 4)
    return {r: torch.cat(v) for r, v in out.items()}


@pytest.mark.parametrize("device,dtype", RUNS)
def test_residual_stream_of_every_layer(mixed_model, device, dtype):
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
    assert len(stream) == len(want) and stream[0].dtype == torch.float32
    for i, (got, exp) in enumerate(zip(stream, want)):
        assert rel(got, exp) < TOL[dtype], f"after layer {i}"


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
    config((latent(), None)), config((delta(), None)), config((delta(1, 1, 16, 8, 1), dense(8)), width=40, vocab=33),
    config((latent(heads=1, dim=4, rot_dim=2, vdim=4, kv_rank=8, q_rank=4), moe(2, 1, 8)), width=70, vocab=65),
    config((latent(heads=9, dim=64, rot_dim=64, vdim=128, kv_rank=256, q_rank=320), moe(9, 4, 200)), (delta(5, 5, 96, 64, 3), moe(3, 3, 48)),
           width=264, vocab=258, eps=1e-3, scale=0.5),
    config((latent(heads=7, dim=56, rot_dim=40, q_rank=24), dense(72)), (delta(8, 2, 112, 48, 5), moe(6, 1, 56)), width=152, vocab=98)],
    ids=["latent only", "delta only", "tiny delta", "tiny latent", "wide", "small query latent"])
def test_other_sizes(cfg, device, dtype):
    t = weights_for(cfg, seed=11)
    toks = torch.randint(0, cfg["vocab"], (90,), generator=torch.Generator().manual_seed(1)).tolist()
    want = oracle.forward(cfg, t, toks)[0]
    out = replay(engine(cfg, t, device, dtype), {"a": toks}, [[("a", n)] for n in (40, 2, 1, 1, 21, 1, 24)])
    assert rel(out["a"], want) < TOL[dtype]


@pytest.mark.parametrize("device,dtype", RUNS)
def test_greedy_generation(device, dtype):
    """More requests than a batch holds through the scheduler, prompts in chunks beside decoding, with preemption when the
    pool runs dry: the tokens are those of plain greedy decoding."""
    cfg = config((latent(), dense()), (delta(), moe()), (latent(kv_from=0), moe(top=1)), vocab=150)
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
    cfg = config((latent(), dense()), (delta(), moe()))
    llm = engine(cfg, weights_for(cfg), "cuda:0", torch.bfloat16, max_logit_rows=0)
    sp = lambda seed: SamplingParams(temperature=1.0, top_k=20, max_new_tokens=16, ignore_eos=True, seed=seed, repetition_penalty=1.2)
    a, b = (llm.generate([[1, 2, 3], [4, 5]], [sp(s), sp(s + 1)]) for s in (5, 9))
    assert all(len(r.tokens) == 16 and 0 <= min(r.tokens) and max(r.tokens) < cfg["vocab"] for r in a + b)
    assert [r.tokens for r in a] != [r.tokens for r in b]


# ---------------------------------------------------------------------------------- configuration, slots, command line
def test_config_checks_and_registry():
    arch = PIPELINE_REGISTRY.retrieve_architecture(MIXED)
    assert arch.name == "Gotunex" and arch.config_class is GotunexConfig
    c = GotunexConfig.from_hf(MIXED)
    assert GotunexConfig.from_hf(c.to_hf()).layers == c.layers and PIPELINE_REGISTRY.retrieve_architecture(c.to_hf()) is arch
    assert c.cache_layers == (0, 2) and c.recurrent_layers == (1, 4)
    with pytest.raises(ValueError):
        GotunexConfig.from_hf(config((latent(), None), (latent(kv_rank=80, kv_from=0), None)))       # another cache row
    with pytest.raises(ValueError):
        GotunexConfig.from_hf(config((latent(), None), (latent(kv_from=0), None), (latent(kv_from=1), None)))
    with pytest.raises(ValueError):
        GotunexConfig.from_hf(config((delta(heads=5, kv_heads=2), None)))
    t = weights_for(MIXED, decay_rank=24, gate_rank=24)
    shapes = c.tensor_shapes()
    assert set(shapes) == set(t)
    assert all(tuple(t[n].shape) == s for n, s in shapes.items() if n.split(".")[-1] not in ("a1", "a2", "g1", "g2"))


def test_state_slots():
    specs = (("s", (3, 2), torch.float32),)
    with pytest.raises(ValueError):
        KVCacheParams(1, 1, 8, 16, torch.float32, True, True, specs)
    p = KVCacheParams(1, 1, 8, 16, torch.float32, True, False, specs)
    kv = PagedKVCacheManager(p, 20, state_slots=2)
    ctx = [TextContext.from_prompt([1] * 20, 64, r) for r in "abc"]
    for c in ctx:
        kv.claim(c)
    assert kv.state_slot_of("a") == -1 and kv.state["s"].shape == (2, 3, 2)
    kv.alloc(ctx[0]), kv.alloc(ctx[1])
    assert {kv.state_slot_of("a"), kv.state_slot_of("b")} == {0, 1}
    assert not kv.can_alloc(ctx[2])
    free = kv.free_blocks
    with pytest.raises(InsufficientBlocksError):
        kv.alloc(ctx[2])
    assert kv.free_blocks == free
    kv.alloc(ctx[0])                                              # a request keeps its slot
    slot = kv.state_slot_of("b")
    kv.release("b")
    kv.alloc(ctx[2])
    assert kv.state_slot_of("c") == slot and kv.free_state_slots == 0
    kv.release("a"), kv.release("c")
    assert kv.free_state_slots == 2


def test_speculation_is_refused():
    from modular_b200.pipelines.speculative import SpeculativeConfig

    with pytest.raises(ValueError):
        engine(config((delta(), None)), weights_for(config((delta(), None))), "cpu", torch.float32,
               speculative=SpeculativeConfig(method="ngram"))


@pytest.mark.parametrize("device,dtype", [RUNS[0], RUNS[1], RUNS[2]])
def test_trace_replay_program(tmp_path, device, dtype):
    """The command-line replay: a checkpoint folder in, steps on standard input, logits in files."""
    cfg = config((latent(), dense()), (delta(), moe()))
    t = weights_for(cfg, seed=31)
    save_checkpoint(str(tmp_path), cfg, {k: v if v.dtype == torch.int32 else v.bfloat16() for k, v in t.items()})
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
