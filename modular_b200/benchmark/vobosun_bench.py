"""Vobosun at sizes that resemble a real model's layers (random weights), beside the closest existing families.

``run_models``: prefill and decode throughput of whole models through the engine's step: Vobosun (softmax-attention and
generalized delta-rule layers in turn, every one followed by experts, with identity experts and a shared one), Mavidra (softmax attention
beside a delta rule, and gated linear attention, in turn) and Gotunex (delta-rule and latent layers) with the same width, heads,
recurrent state sizes and experts.
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
from .mavidra_bench import SIZES, gotunex_config

GROUPS, KEEP = 8, 4


def vobosun_config(s: dict):
    from ..models.vobosun import VobosunConfig

    d = s["dim"]
    att = dict(heads=s["heads"], kv_heads=s["kv_heads"], dim=d, vdim=d, scale=d ** -0.5,
               rot=dict(base=500000.0, dims=d // 2, scaling=dict(factor=4.0)))
    router = dict(experts=s["experts"], top=s["top"], identity=GROUPS, groups=dict(count=GROUPS, keep=KEEP))
    return VobosunConfig.build(s["width"], s["vocab"], "".join("ME"[i % 2] for i in range(s["layers"])), att, dict(heads=s["rheads"], dim=s["rdim"]),
                               0, s["expert_ff"], router, s["expert_ff"])


def mavidra_config(s: dict):
    """The same attention heads, recurrent states and experts; its softmax layers have a delta rule beside them."""
    from ..models.mavidra import MavidraConfig

    d, e = s["dim"], s["rdim"]
    left = dict(heads=s["heads"], kv_heads=s["kv_heads"], dim=d, vdim=d, scale=d ** -0.5, rot=dict(base=500000.0, dims=d // 2))
    right = dict(heads=s["rheads"], kv_heads=s["rheads"], dim=e, vdim=e, conv=4)
    return MavidraConfig.build(s["width"], s["vocab"], "".join("PG"[i % 2] for i in range(s["layers"])),
                               dict(heads=s["rheads"], dim=e, vdim=e, tau=16.0), {}, dict(left=left, right=right, left_scale=0.5, right_scale=0.5),
                               s["expert_ff"], dict(experts=s["experts"], top=s["top"], groups=dict(count=GROUPS, keep=KEEP)),
                               dict(buckets=s["vocab"], mul_prev=65537, mul_cur=31))


def run_models(sizes=tuple(SIZES), prefill=2048, seqs=4, batches=(1, 64), context=2048, steps=20):
    """Yields one record per (size, model, decode batch)."""
    import gc

    for name in sizes:
        s = SIZES[name]
        for label, cfg in (("vobosun", vobosun_config(s)), ("mavidra (softmax beside delta, gated linear)", mavidra_config(s)),
                           ("gotunex (delta + latent, experts)", gotunex_config(s))):
            for batch in batches:
                r = bench_engine(cfg, prefill, seqs, batch, context, steps)
                yield {"size": name, "model": label, "layers": s["layers"], **r}
                gc.collect()
                torch.cuda.empty_cache()


def run_kernels(s: dict, name: str, prefill: int = 2048, seqs: int = 4, batch: int = 64, context: int = 2048) -> list:
    """Every kernel of the design beside the like kernel of an existing family, same shapes, L2 flushed."""
    from ..nn.delta_rule import DeltaRule, DeltaRuleConfig, delta_rule_cuda
    from ..nn.general_delta import GeneralDelta, GeneralDeltaConfig
    from ..nn.residual import sandwich_norm, tanh_seam
    from ..nn.rotary_embedding import cos_sin_table
    from ..nn.window_attention import block_prep, tensor_core_plan, window_attention

    peaks, rows, L = measured_peaks(), [], lib()
    bf = lambda *shape: torch.randn(*shape, device="cuda").bfloat16()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    W, H, KH, d, page = s["width"], s["heads"], s["kv_heads"], s["dim"], 128
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
        seen = (ctx if one else ctx * (ctx + 1) // 2) * B
        # --- softmax attention
        kv = bf(B * n_pages, 2, 1, KH, page, d)
        px, o = bf(T, (H + 2 * KH) * d), torch.empty(T, H * d, device="cuda", dtype=torch.bfloat16)
        q = px[:, : H * d]
        plan, lplan = tensor_core_plan(H // KH, d, torch.bfloat16, page, qs, ql, T, one), tuple(
            torch.from_numpy(a).cuda() if a.size else None for a in ops.build_attention_plan(ql.cpu().numpy(), H, KH))
        add("softmax attention", "paged_attention", phase, lambda: window_attention(q, kv, 0, bt, qs, ql, kl, H, KH, d ** -0.5, 0, None, plan, o),
            lambda: ops.paged_attention(q, kv[:, 0, 0], kv[:, 1, 0], bt, qs, ql, kl, H, KH, d, d ** -0.5, lplan, o, kv, 0),
            2.0 * (2 * T * H * d + 2 * B * ctx * KH * d), 4.0 * seen * H * d)
        # --- biases, rotation and the store, beside rotation and store
        rot, bias = d // 2, torch.randn((H + 2 * KH) * d, device="cuda")
        cs, lcs = cos_sin_table(rot, ctx + 1, 1e4, None, "cuda"), cos_sin_table(d, ctx + 1, 1e4, None, "cuda")
        add("block_prep (biases)", "rope_kv_store", phase,
            lambda: block_prep(px, H, H * d, (H + KH) * d, KH, rot, pos, cs, slots, kv, 0, halves=True, bias=bias),
            lambda: ops.rope_kv_store(px, pos, slots, lcs, kv[:, 0, 0], kv[:, 1, 0], H, KH, d), 4.0 * T * (H + 2 * KH) * d)
        del kv, px, o, q
        # --- seams
        x, y, a, n1, own = torch.randn(T, W, device="cuda"), torch.empty(T, W, device="cuda"), bf(T, W), bf(T, W), bf(T, W)
        w1, b1, w2, b2, mix, prev = bf(W), bf(W), bf(W), bf(W), bf(W), torch.zeros(B, W, device="cuda")
        shift = dict(shift=mix, prev=prev, state_idx=idx, q_start=qs, q_len=ql, kv_len=kl_new)
        like = lambda: sandwich_norm(x, a=a, w_u=w2, b_u=b2, mult=0.5, w1=w1, b1=b1, n1=n1)
        by = T * W * (8.0 + 2.0 + 2.0)
        add("tanh_seam", "sandwich_norm", phase, lambda: tanh_seam(x=x, x_out=x, a=a, norm_u=(0.5, w2, b2), norm1=(0.5, w1, b1), n1=n1), like, by)
        add("tanh_seam (token shift)", "sandwich_norm", phase,
            lambda: tanh_seam(x=x, x_out=y, a=a, norm_u=(0.5, w2, b2), norm1=(0.5, w1, b1), n1=n1, **shift), like, by + B * W * (8.0 if one else 4.0),
            like_bytes=by)
        # --- experts: choice and order, and the seam that adds their outputs (an eighth of the pairs are identity experts)
        logits, corr = torch.randn(T, E + GROUPS, device="cuda"), torch.randn(E + GROUPS, device="cuda")
        int_ = lambda *shape: torch.empty(*shape, dtype=torch.int32, device="cuda")
        ids, rank, inv, offs, counts = int_(T, k), int_(T, k), int_(T, k), int_(E + 1), int_(E)
        pw, place, eo = torch.empty(T, k, device="cuda"), bf(T * k, W), bf(T * k, W)

        def route(identity, softmax):
            counts.zero_()
            L.moe_score_route(logits[:, : E + identity], corr, ids, pw, rank, counts, GROUPS, KEEP, softmax, 1.0, softmax, softmax, identity)
            L.moe_place_rows(n1, ids, rank, counts, offs, inv, place)

        add("router (softmax, identity) + place_rows", "router (sigmoid) + place_rows", phase, lambda: route(GROUPS, True), lambda: route(0, False),
            T * (4.0 * E + 2.0 * W * (1 + k)))
        route(0, False)
        linv = inv.clone()
        route(GROUPS, True)
        share = float((inv >= 0).float().mean())
        add("tanh_seam (experts, shared, shift)", "sandwich_norm (experts)", phase,
            lambda: tanh_seam(x=x, x_out=y, a=a, e=eo, inverse=inv, pair_w=pw, self_rows=own, norm_u=(0.5, w2, b2), norm1=(0.5, w1, b1), n1=n1, **shift),
            lambda: sandwich_norm(x, e=eo, inverse=linv, pair_w=pw, w_u=w2, b_u=b2, mult=0.5, w1=w1, b1=b1, n1=n1),
            T * W * (8.0 + 2.0 * k * share + 2.0 + 2.0 + 2.0), like_bytes=T * W * (8.0 + 2.0 * k + 2.0))
        del eo, place, x, y, a
        # --- activations
        ff = bf(T, s["expert_ff"] * 2)
        add("xielu", "gelu_tanh", phase, lambda: ops.xielu(ff, 0.7, 1.1), lambda: ops.gelu_tanh(ff), 4.0 * ff.numel())
        low = bf(T, 64)
        add("tanh (64 columns)", "gelu_tanh", phase, lambda: ops.tanh(low), lambda: ops.gelu_tanh(low), 4.0 * low.numel())
        # --- recurrence, beside the delta rule with a decay per channel
        lc = DeltaRuleConfig(W, h, h, e, e, 4, e, e, 1e-6)
        lm = DeltaRule.__new__(DeltaRule)
        lm.cfg, lm.off = lc, {n: at for n, _, at in lc.blocks}
        lm.conv_w, lm.norm, lm.A_log, lm.dt_bias = bf(lc.channels, 4), bf(e), torch.zeros(h, device="cuda"), torch.zeros(h * e, device="cuda")
        lx = bf(T, -(-(lc.blocks[-1][2] + lc.blocks[-1][1]) // 8) * 8)
        z, g, out = torch.randn(T, h * e, device="cuda"), bf(T, h * e), bf(T, h * e)
        st, cv = (torch.zeros(B, *sh, device="cuda") for sh in (lc.state_shapes()["delta"], lc.state_shapes()["conv"]))
        gm = GeneralDelta.__new__(GeneralDelta)
        gm.cfg = GeneralDeltaConfig(h, e, 64, 1e-6)
        gm.k_off, gm.v_off, gm.g_off, gm.a_off, gm.w_off = (i * h * e for i in range(1, 6))
        gm.a_bias, gm.w_bias, gm.norm, gx = torch.zeros(h * e, device="cuda"), torch.zeros(h * e, device="cuda"), bf(h * e), bf(T, 5 * h * e)
        state = B * h * e * e * 4.0 * (2 if one else 1)
        add("generalized delta rule", "delta rule", phase, lambda: gm.mix(gx, z, out, st, idx, qs, ql, kl_new, one),
            lambda: delta_rule_cuda(lm, lx, z, g, out, st, cv, idx, qs, ql, kl_new, one), T * h * e * (10.0 + 4.0 + 2.0) + state, 10.0 * T * h * e * e,
            FP32_TFLOPS, T * (lx.shape[1] * 2.0 + h * e * 8) + state, 9.0 * T * h * e * e)
        del lx, gx, st, cv, z, g, out
        torch.cuda.empty_cache()
    return rows


def main(sizes=tuple(SIZES), steps: int = 20) -> dict:
    return {"peaks": measured_peaks(), "fp32_tflops_nominal": FP32_TFLOPS, "kernels": [r for n in sizes for r in run_kernels(SIZES[n], n)],
            "models": list(run_models(sizes, steps=steps))}
