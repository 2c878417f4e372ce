"""Mavidra at sizes that resemble a real model's layers (random weights), beside the closest existing families.

``run_models``: prefill and decode throughput of whole models through the engine's step: Mavidra (gated linear, latent and
parallel layers in turn) and Gotunex (delta-rule and latent layers) with the same width, heads, latents, recurrent state sizes
and experts, every layer of both followed or accompanied by experts.
``run_kernels``: every kernel of the design beside the like kernel of an existing family on the same shapes, with its distance
from a roofline (measured copy bandwidth and GEMM rate; the nominal fp32 rate for recurrences on the CUDA cores).
"""

from __future__ import annotations

import torch

from .. import ops
from .._native import lib
from ..utils.peaks import measured_peaks
from .gotunex_bench import FP32_TFLOPS, bench_engine
from .kernel_bench import time_fn

SIZES = {
    # width, layers, attention heads, kv heads, head width, latent ranks, window, recurrent heads and widths, experts
    "w2048": dict(width=2048, layers=12, heads=16, kv_heads=4, dim=128, kv_rank=512, q_rank=1536, window=1024, rheads=16, rdim=128,
                  experts=64, top=6, expert_ff=1408, vocab=102400),
    "w4096": dict(width=4096, layers=8, heads=32, kv_heads=8, dim=128, kv_rank=512, q_rank=1536, window=1024, rheads=32, rdim=128,
                  experts=32, top=4, expert_ff=2048, vocab=128256),
    "w7168": dict(width=7168, layers=4, heads=128, kv_heads=8, dim=128, kv_rank=512, q_rank=1536, window=1024, rheads=64, rdim=128,
                  experts=32, top=4, expert_ff=2048, vocab=129280),
}


def mavidra_config(s: dict):
    from ..models.mavidra import MavidraConfig

    d, e = s["dim"], s["rdim"]
    latent = dict(heads=s["heads"], dim=d, rot_dim=64, vdim=d, kv_rank=s["kv_rank"], q_rank=s["q_rank"], scale=(d + 64) ** -0.5,
                  mask=dict(size=s["window"]), rot=dict(base=10000.0, dims=64))
    left = dict(heads=s["heads"], kv_heads=s["kv_heads"], dim=d, vdim=d, scale=d ** -0.5, rot=dict(base=500000.0, dims=d // 2))
    right = dict(heads=s["rheads"], kv_heads=s["rheads"], dim=e, vdim=e, conv=4)
    pattern = "".join("GAPS"[i % 4] for i in range(s["layers"]))
    return MavidraConfig.build(s["width"], s["vocab"], pattern, dict(heads=s["rheads"], dim=e, vdim=e, tau=16.0), latent,
                               dict(left=left, right=right, left_scale=0.5, right_scale=0.5), s["expert_ff"],
                               dict(experts=s["experts"], top=s["top"], groups=dict(count=8, keep=4)),
                               dict(buckets=s["vocab"], mul_prev=65537, mul_cur=31))


def gotunex_config(s: dict):
    """The same latents, recurrent state sizes and experts: a delta-rule layer for every gated linear and parallel one."""
    from ..models.gotunex import GotunexConfig

    d, e = s["dim"], s["rdim"]
    att = dict(heads=s["heads"], dim=d, rot_dim=64, vdim=d, kv_rank=s["kv_rank"], q_rank=s["q_rank"], scale=(d + 64) ** -0.5,
               rot=dict(base=10000.0, dims=64))
    delta = dict(heads=s["rheads"], kv_heads=s["rheads"], dim=e, vdim=e, conv=4)
    return GotunexConfig.build(s["width"], s["vocab"], "".join("DADS"[i % 4] for i in range(s["layers"])), att, delta, 0, s["expert_ff"],
                               s["experts"], s["top"])


def run_models(sizes=tuple(SIZES), prefill=2048, seqs=4, batches=(1, 64), context=2048, steps=20):
    """Yields one record per (size, model, decode batch)."""
    import gc

    for name in sizes:
        s = SIZES[name]
        for label, cfg in (("mavidra", mavidra_config(s)), ("gotunex (delta + latent, experts)", gotunex_config(s))):
            for batch in batches:
                r = bench_engine(cfg, prefill, seqs, batch, context, steps)
                yield {"size": name, "model": label, "layers": s["layers"], **r}
                gc.collect()
                torch.cuda.empty_cache()


def run_kernels(s: dict, name: str, prefill: int = 2048, seqs: int = 4, batch: int = 64, context: int = 2048) -> list:
    """Every kernel of the design beside the like kernel of an existing family, same shapes, L2 flushed."""
    from ..nn.bigram import BigramConfig, bigram_rows
    from ..nn.delta_rule import DeltaRule, DeltaRuleConfig, delta_rule_cuda
    from ..nn.gated_linear_attention import GatedLinearAttention, GatedLinearConfig
    from ..nn.latent_attention import latent_attention
    from ..nn.moe import TableRouter
    from ..nn.residual import residual_norm, sandwich_norm
    from ..nn.rotary_embedding import cos_sin_table
    from ..nn.window_attention import block_prep, tensor_core_plan, window_attention

    peaks, rows, L = measured_peaks(), [], lib()
    bf = lambda *shape: torch.randn(*shape, device="cuda").bfloat16()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    W, H, KH, d, R, window, page = s["width"], s["heads"], s["kv_heads"], s["dim"], s["kv_rank"], s["window"], 128
    h, e, E, k = s["rheads"], s["rdim"], s["experts"], s["top"]

    def add(kernel, like, phase, fn, like_fn, nbytes, flops=0.0, tflops=None, like_bytes=None, like_flops=None, like_tflops=None):
        roof = lambda b, f, peak: max(b / (peaks["hbm_gbs"] * 1e9), f / ((peak or peaks["bf16_tflops"]) * 1e12))
        t, u = time_fn(fn), time_fn(like_fn)
        rows.append({"size": name, "kernel": kernel, "phase": phase, "us": t * 1e6, "frac_of_roofline": roof(nbytes, flops, tflops) / t,
                     "like": like, "like_us": u * 1e6,
                     "like_frac": roof(nbytes if like_bytes is None else like_bytes, flops if like_flops is None else like_flops,
                                       like_tflops or tflops) / u})

    for phase, T, B, ctx in (("prefill", prefill * seqs, seqs, prefill), ("decode", batch, batch, context), ("decode b1", 1, 1, context)):
        one = T == B
        ql, kl = i32([T // B] * B), i32([ctx] * B)
        qs, pos = (torch.cumsum(ql, 0) - ql).int(), torch.arange(T, device="cuda", dtype=torch.int32) % ctx
        if one:
            pos = kl - 1
        kl_new, idx = (kl if one else ql), torch.arange(B, device="cuda", dtype=torch.int32)
        n_pages = -(-ctx // page)
        bt = torch.randperm(B * n_pages, device="cuda").int().view(B, n_pages)
        slots = bt.repeat_interleave(T // B, 0)[torch.arange(T, device="cuda"), pos.long() // page].long() * page + pos.long() % page
        seen = lambda w: (min(w, ctx) if one else sum(min(i + 1, w) for i in range(ctx))) * B
        keys = lambda w: B * min(ctx, w if one else ctx)
        # --- latent attention: a window and a gate, beside the whole context with a sink
        cache, gate = bf(B * n_pages, page, R + 64), bf(T, H)
        q_lat, q_rope, sink = bf(T, H, R), bf(T, H, 64), torch.randn(H, device="cuda")
        cost = lambda w: (2.0 * (T * H * (2 * R + 64) + keys(w) * (R + 64)), 2.0 * seen(w) * H * (2 * R + 64))
        (by, fl), (lby, lfl) = cost(window), cost(1 << 30)
        add("latent attention (window, gate)", "latent attention (sink)", phase,
            lambda: latent_attention(q_lat, q_rope, cache, bt, qs, ql, kl, 0.1, None, one, window, gate),
            lambda: latent_attention(q_lat, q_rope, cache, bt, qs, ql, kl, 0.1, sink, one), by, fl, None, lby, lfl)
        del cache, q_lat, q_rope
        # --- softmax attention: a sink and a gate, beside plain grouped attention
        kv = bf(B * n_pages, 2, 1, KH, page, d)
        px, o = bf(T, (H + 2 * KH) * d), torch.empty(T, H * d, device="cuda", dtype=torch.bfloat16)
        q = px[:, : H * d]
        plan, lplan = tensor_core_plan(H // KH, d, torch.bfloat16, page, qs, ql, T, one), tuple(
            torch.from_numpy(a).cuda() if a.size else None for a in ops.build_attention_plan(ql.cpu().numpy(), H, KH))
        by, fl = 2.0 * (2 * T * H * d + 2 * keys(1 << 30) * KH * d), 4.0 * seen(1 << 30) * H * d
        add("softmax attention (sink, gate)", "paged_attention", phase,
            lambda: window_attention(q, kv, 0, bt, qs, ql, kl, H, KH, d ** -0.5, 0, sink, plan, o, gate, 0.5),
            lambda: ops.paged_attention(q, kv[:, 0, 0], kv[:, 1, 0], bt, qs, ql, kl, H, KH, d, d ** -0.5, lplan, o, kv, 0), by, fl)
        # --- norms and rotation of queries and keys, and the store
        rot, qn, kn = d // 2, bf(d), bf(d)
        cs, lcs = cos_sin_table(rot, ctx + 1, 1e4, None, "cuda"), cos_sin_table(d, ctx + 1, 1e4, None, "cuda")

        def like_prep():
            ops.qk_norm(px, qn, kn, H, KH, d, 1e-6)
            ops.rope_kv_store(px, pos, slots, lcs, kv[:, 0, 0], kv[:, 1, 0], H, KH, d)

        add("block_prep (head norms)", "qk_norm + rope_kv_store", phase,
            lambda: block_prep(px, H, H * d, (H + KH) * d, KH, rot, pos, cs, slots, kv, 0, q_norm=qn, k_norm=kn, norm_dim=d, halves=True), like_prep,
            4.0 * T * (H + 2 * KH) * d)
        del kv, px, o, q
        # --- seams: one branch with a norm on both sides, beside two branches and two norms
        x, a, b, n1, n2 = torch.randn(T, W, device="cuda"), bf(T, W), bf(T, W), bf(T, W), bf(T, W)
        w1, b1, w2, b2 = bf(W), bf(W), bf(W), bf(W)
        add("sandwich_norm", "residual_norm", phase, lambda: sandwich_norm(x, a=a, w_u=w2, b_u=b2, mult=0.5, w1=w1, b1=b1, n1=n1),
            lambda: residual_norm(x, a=a, b=b, w1=w1, n1=n1, w2=w2, n2=n2), T * W * (8.0 + 2.0 + 2.0), like_bytes=T * W * 16.0)
        # --- experts: choice and order, and the seam that adds their outputs; beside the kernels of the other families
        logits, corr = torch.randn(T, E, device="cuda"), torch.randn(E, device="cuda")
        int_ = lambda *shape: torch.empty(*shape, dtype=torch.int32, device="cuda")
        ids, rank, inv, offs, counts = int_(T, k), int_(T, k), int_(T, k), int_(E + 1), int_(E)
        pw, place, eo = torch.empty(T, k, device="cuda"), bf(T * k, W), bf(T * k, W)
        scratch, order, inv2 = torch.zeros(2 * E, dtype=torch.int32, device="cuda"), int_(T * k), int_(T * k)
        groups, keep = 8, 4

        def route():
            counts.zero_()
            L.moe_score_route(logits, corr, ids, pw, rank, counts, groups, keep, False, 1.0)
            L.moe_place_rows(n1, ids, rank, counts, offs, inv, place)

        def like_route():
            L.moe_router_group_limited(logits, corr, ids, pw, groups, keep, False, 1.0)
            L.moe_create_indices(ids, 0, E, scratch, offs, order, inv2)
            L.moe_permute_rows(n1, order, offs[E:], place, k)

        add("moe_score_route + place_rows", "router + create_indices + permute", phase, route, like_route, T * (4.0 * E + 2.0 * W * (1 + k)))
        route()
        add("sandwich_norm (experts)", "residual_norm (experts)", phase,
            lambda: sandwich_norm(x, e=eo, inverse=inv, pair_w=pw, w_u=w2, b_u=b2, mult=0.5, w1=w1, b1=b1, n1=n1),
            lambda: residual_norm(x, a=a, e=eo, inverse=inv, pair_w=1 / k, w1=w1, n1=n1, w2=w2, n2=place, scatter=inv),
            T * W * (8.0 + 2.0 * k + 2.0), like_bytes=T * W * (8.0 + 2.0 + 2.0 * k + 2.0 + 2.0 * k))
        del eo, place, x, a, b
        # --- recurrences, beside the delta rule with a decay per channel
        lc = DeltaRuleConfig(W, h, h, e, e, 4, e, e, 1e-6)
        nc = DeltaRuleConfig(W, h, h, e, e, 4, 0, 0, 1e-6, head_decay=True, out_mult=0.5)

        def delta(c):
            m = DeltaRule.__new__(DeltaRule)
            m.cfg, m.off = c, {n: at for n, _, at in c.blocks}
            m.conv_w, m.norm, m.A_log = bf(c.channels, 4), bf(e), torch.zeros(h, device="cuda")
            m.dt_bias = torch.zeros(h if c.head_decay else h * e, device="cuda")
            rows_ = c.blocks[-1][2] + c.blocks[-1][1]
            return m, bf(T, -(-rows_ // 8) * 8)

        (lm, lx), (nm, nx) = delta(lc), delta(nc)
        z, g, out = torch.randn(T, h * e, device="cuda"), bf(T, h * e), bf(T, h * e)
        st, cv = (torch.zeros(B, *sh, device="cuda") for sh in (lc.state_shapes()["delta"], lc.state_shapes()["conv"]))
        state = B * h * e * e * 4.0 * (2 if one else 1)
        like = lambda: delta_rule_cuda(lm, lx, z, g, out, st, cv, idx, qs, ql, kl_new, one)
        lby, lfl = T * (lx.shape[1] * 2.0 + h * e * 8) + state, 9.0 * T * h * e * e
        add("delta rule (decay per head)", "delta rule", phase,
            lambda: delta_rule_cuda(nm, nx, None, nx[:, nm.off["g"]: nm.off["g"] + h * e], out, st, cv, idx, qs, ql, kl_new, one), like,
            T * (nx.shape[1] * 2.0 + h * e * 2) + state, lfl, FP32_TFLOPS, lby, lfl)
        gm = GatedLinearAttention.__new__(GatedLinearAttention)
        gm.cfg = GatedLinearConfig(h, e, e, 16, 16.0, 1e-6)
        gm.k_off, gm.v_off, gm.g_off, gm.a_off = h * e, 2 * h * e, 3 * h * e, 4 * h * e
        gm.a_bias, gm.norm, gx = torch.zeros(h * e, device="cuda"), bf(e), bf(T, 4 * h * e)
        add("gated linear attention", "delta rule", phase, lambda: gm.mix(gx, z, out, st, idx, qs, ql, kl_new, one), like,
            T * h * e * (8.0 + 4.0 + 2.0) + state, 5.0 * T * h * e * e, FP32_TFLOPS, lby, lfl)
        # --- bigram rows, beside the other kernel that turns token ids into row numbers (one layer's experts)
        toks, last = torch.randint(0, 1000, (T,), device="cuda"), torch.zeros(B, 1, dtype=torch.int64, device="cuda")
        bc, table = BigramConfig(1009, 31, 7), TableRouter([torch.rand(1000, E).topk(1, -1).indices.int()], [E], "cuda")
        add("bigram_rows", "moe_table_route (1 layer, top 1)", phase, lambda: bigram_rows(bc, toks, qs, ql, kl_new, idx, last),
            lambda: table.route(toks), 16.0 * T)
        del lx, nx, gx, st, cv, z, g, out
        torch.cuda.empty_cache()
    return rows


def main(sizes=tuple(SIZES), steps: int = 20) -> dict:
    return {"peaks": measured_peaks(), "fp32_tflops_nominal": FP32_TFLOPS, "kernels": [r for n in sizes for r in run_kernels(SIZES[n], n)],
            "models": list(run_models(sizes, steps=steps))}
