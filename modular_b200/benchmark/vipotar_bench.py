"""Vipotar at sizes that resemble a real model's layers (random weights), beside the closest existing families.

``run_models``: prefill and decode throughput of whole models through the engine's step: Vipotar (some layers looped), Gotunex
(delta-rule and latent-attention layers, the other family with recurrent state and an fp32 stream) and Llama, with as many
layers as Vipotar has layer runs and feed-forwards chosen for equal weights per layer.
``run_kernels``: every kernel of the design beside the like kernel of an existing family on the same shapes, with its distance
from a roofline (measured copy bandwidth and GEMM rate; the nominal fp32 rate for the delta rule).
"""

from __future__ import annotations

import torch

from .. import ops
from .._native import lib
from ..utils.peaks import measured_peaks
from .gotunex_bench import FP32_TFLOPS, bench_engine
from .kernel_bench import time_fn

SIZES = {
    "w2048": dict(width=2048, layers=10, loop=(2, 5, 2), heads=16, kv_heads=4, dim=128, window=1024, rheads=16, rdim=128, ff=8192, vocab=102400),
    "w4096": dict(width=4096, layers=6, loop=(2, 4, 2), heads=32, kv_heads=8, dim=128, window=1024, rheads=32, rdim=128, ff=14336, vocab=128256),
    "w8192": dict(width=8192, layers=3, loop=(1, 2, 2), heads=64, kv_heads=8, dim=128, window=4096, rheads=64, rdim=128, ff=28672, vocab=128256),
}


def vipotar_config(s: dict):
    from ..models.vipotar import VipotarConfig

    d, (a, b, n) = s["dim"], s["loop"]
    left = dict(heads=s["heads"], kv_heads=s["kv_heads"], dim=d, vdim=d, scale=d ** -0.5, mask={"size": s["window"]},
                rot=dict(base=500000.0, dims=d // 2, scaling=dict(factor=8.0, original=8192, fast=32.0, slow=1.0)))
    return VipotarConfig.build(s["width"], s["vocab"], s["layers"], left, dict(heads=s["rheads"], dim=s["rdim"], vdim=s["rdim"]), s["ff"],
                               {"start": a, "stop": b, "times": n})


def layer_weights(s: dict) -> int:
    """Weights of one Vipotar layer's projections."""
    W, d, e = s["width"], s["dim"], s["rheads"] * s["rdim"]
    return W * (2 * s["heads"] * d + 2 * s["kv_heads"] * d + 5 * e + 2 * s["ff"])


def runs(s: dict) -> int:
    a, b, n = s["loop"]
    return s["layers"] + (b - a) * (n - 1)


def llama_config(s: dict):
    """As many layers as Vipotar has runs, each with its attention and the weights of its other projections in the SwiGLU."""
    from ..models.llama3 import Llama3Config

    W, q, kv = s["width"], s["heads"] * s["dim"], s["kv_heads"] * s["dim"]
    ff = (layer_weights(s) - 2 * W * (q + kv)) // (3 * W) // 256 * 256
    return Llama3Config(hidden_size=W, intermediate_size=ff, num_hidden_layers=runs(s), num_attention_heads=s["heads"],
                        num_key_value_heads=s["kv_heads"], head_dim=s["dim"], vocab_size=s["vocab"])


def gotunex_config(s: dict):
    """Delta-rule and latent-attention layers in turn, dense feed-forwards that even out the weights per layer."""
    from ..models.gotunex import GotunexConfig

    W, e, d = s["width"], s["rheads"] * s["rdim"], s["dim"]
    att = dict(heads=s["heads"], dim=d, rot_dim=64, vdim=d, kv_rank=512, q_rank=1536, scale=(d + 64) ** -0.5, rot=dict(base=10000.0, dims=64))
    delta = dict(heads=s["rheads"], kv_heads=s["rheads"], dim=s["rdim"], vdim=s["rdim"], conv=4)
    ff = (layer_weights(s) - 4 * W * e) // (2 * W) // 256 * 256
    return GotunexConfig.build(W, s["vocab"], "".join("da"[i % 2] for i in range(runs(s))), att, delta, ff, 0, 0, 0)


def run_models(sizes=tuple(SIZES), prefill=2048, seqs=4, batches=(1, 64), context=2048, steps=20):
    """Yields one record per (size, model, decode batch)."""
    import gc

    for name in sizes:
        s = SIZES[name]
        for label, cfg in (("vipotar", vipotar_config(s)), ("gotunex (delta + latent, dense)", gotunex_config(s)), ("llama", llama_config(s))):
            for batch in batches:
                r = bench_engine(cfg, prefill, seqs, batch, context, steps)
                yield {"size": name, "model": label, "layers": runs(s), **r}
                gc.collect()
                torch.cuda.empty_cache()


def run_kernels(s: dict, name: str, prefill: int = 2048, seqs: int = 4, batch: int = 64, context: int = 2048) -> list:
    """Every kernel of the design beside the like kernel of an existing family, same shapes, L2 flushed."""
    from ..nn.delta_rule import DeltaRule, DeltaRuleConfig, delta_rule_cuda
    from ..nn.residual import residual_norm
    from ..nn.rotary_embedding import cos_sin_table
    from ..nn.window_attention import block_prep, tensor_core_plan, window_attention

    peaks, rows, L = measured_peaks(), [], lib()
    bf = lambda *shape: torch.randn(*shape, device="cuda").bfloat16()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    W, H, KH, d, F, page = s["width"], s["heads"], s["kv_heads"], s["dim"], s["ff"], 128
    h, e, window = s["rheads"], s["rdim"], s["window"]
    n_in = (H + 2 * KH) * d + 4 * h * e + F

    def add(kernel, like, phase, fn, like_fn, nbytes, flops=0.0, like_bytes=None, like_flops=None, like_tflops=None):
        roof = lambda b, f, peak=None: max(b / (peaks["hbm_gbs"] * 1e9), f / ((peak or peaks["bf16_tflops"]) * 1e12))
        t, u = time_fn(fn), time_fn(like_fn)
        rows.append({"size": name, "kernel": kernel, "phase": phase, "us": t * 1e6, "frac_of_roofline": roof(nbytes, flops) / t, "like": like,
                     "like_us": u * 1e6, "like_frac": roof(nbytes if like_bytes is None else like_bytes,
                                                           flops if like_flops is None else like_flops, like_tflops) / u})

    for phase, T, B, ctx in (("prefill", prefill * seqs, seqs, prefill), ("decode", batch, batch, context), ("decode b1", 1, 1, context)):
        one = T == B
        ql, kl = i32([T // B] * B), i32([ctx] * B)
        qs, pos = (torch.cumsum(ql, 0) - ql).int(), torch.arange(T, device="cuda", dtype=torch.int32) % ctx
        if one:
            pos = kl - 1
        n_pages = -(-ctx // page)
        kv = torch.randn(B * n_pages, 2, 1, KH, page, d, device="cuda").bfloat16()
        bt = torch.randperm(B * n_pages, device="cuda").int().view(B, n_pages)
        slots = bt.repeat_interleave(T // B, 0)[torch.arange(T, device="cuda"), pos.long() // page].long() * page + pos.long() % page
        px, sink = bf(T, n_in), torch.zeros(H, device="cuda")
        q, o = px[:, : H * d], torch.empty(T, H * d, device="cuda", dtype=torch.bfloat16)
        # --- attention: a window and a sink, beside the same heads over the whole context
        seen = lambda w: (min(w, ctx) if one else sum(min(i + 1, w) for i in range(ctx))) * B
        keys = lambda w: B * min(ctx, w if one else ctx)
        cost = lambda w: (2.0 * (2 * T * H * d + 2 * keys(w) * KH * d), 4.0 * seen(w) * H * d)
        plan, lplan = tensor_core_plan(H // KH, d, torch.bfloat16, page, qs, ql, T, one), tuple(
            torch.from_numpy(a).cuda() if a.size else None for a in ops.build_attention_plan(ql.cpu().numpy(), H, KH))
        (by, fl), (lby, lfl) = cost(window), cost(1 << 30)
        add("window attention (sink)", "paged_attention", phase,
            lambda: window_attention(q, kv, 0, bt, qs, ql, kl, H, KH, d ** -0.5, window, sink, plan, o),
            lambda: ops.paged_attention(q, kv[:, 0, 0], kv[:, 1, 0], bt, qs, ql, kl, H, KH, d, d ** -0.5, lplan, o, kv, 0), by, fl, lby, lfl)
        # --- between the input projection and the branches, beside the rotation + store and the SwiGLU product
        rot = d // 2
        cs, lcs = cos_sin_table(rot, ctx + 1, 1e4, None, "cuda"), cos_sin_table(d, ctx + 1, 1e4, None, "cuda")
        ro, up = (H + 2 * KH) * d, n_in - F
        gu, act = bf(T, 2 * F), torch.empty(T, F, device="cuda", dtype=torch.bfloat16)

        def like_prep():
            ops.rope_kv_store(px, pos, slots, lcs, kv[:, 0, 0], kv[:, 1, 0], H, KH, d)
            ops.silu_mul(gu, act)

        add("block_prep", "rope_kv_store + silu_mul", phase,
            lambda: block_prep(px, H, H * d, (H + KH) * d, KH, rot, pos, cs, slots, kv, 0, (ro, 3 * h * e), (up, F)), like_prep,
            4.0 * T * (H * rot + 2 * KH * d + 3 * h * e + F), like_bytes=T * (4.0 * (H + 2 * KH) * d + 6.0 * F))
        px.normal_()
        # --- seam: two normed branches, the feed-forward, one norm; beside the seam of Gotunex (two branches, two norms)
        x, a, b, c, n1, n2 = torch.randn(T, W, device="cuda"), bf(T, W), bf(T, W), bf(T, W), bf(T, W), bf(T, W)
        w1, w2, w3 = bf(W), bf(W), bf(W)
        add("residual_norm (branch norms)", "residual_norm", phase,
            lambda: residual_norm(x, a=a, b=b, norm_a=w2, norm_b=w3, ab_scale=0.5, c=c, mult=0.5, w1=w1, n1=n1),
            lambda: residual_norm(x, a=a, b=b, w1=w1, n1=n1, w2=w2, n2=n2), T * W * (8.0 + 6.0 + 2.0), like_bytes=T * W * 16.0)
        # --- recurrence, beside the delta rule of the same heads
        xr = px[:, ro: up]
        st = torch.zeros(B, h, e, e, device="cuda")
        decay = torch.full((h,), 0.95, device="cuda")
        powers = decay.unsqueeze(1) ** torch.arange(65, device="cuda")
        idx, ro_o = torch.arange(B, device="cuda", dtype=torch.int32), torch.empty(T, h * e, device="cuda", dtype=torch.bfloat16)
        state = B * h * e * e * 4.0 * (2 if one else 1)
        lc = DeltaRuleConfig(W, h, h, e, e, 4, e, e, 1e-6)
        m = DeltaRule.__new__(DeltaRule)
        m.cfg, m.off = lc, {n: at for n, _, at in lc.blocks}
        pxd = bf(T, lc.blocks[-1][2] + lc.blocks[-1][1])
        m.conv_w, m.A_log, m.dt_bias, m.norm = bf(lc.channels, 4), torch.zeros(h, device="cuda"), torch.zeros(h * e, device="cuda"), bf(e)
        z, gate, lo = torch.randn(T, h * e, device="cuda"), bf(T, h * e), bf(T, h * e)
        lst, lcv = (torch.zeros(B, *sh, device="cuda") for sh in (lc.state_shapes()["delta"], lc.state_shapes()["conv"]))
        kl_new = kl if one else ql
        add("lightning", "delta rule", phase,
            lambda: L.lightning(xr, 0, h * e, 2 * h * e, decay, powers, ro_o, st, idx, qs, ql, kl_new, h, e, e, one),
            lambda: delta_rule_cuda(m, pxd, z, gate, lo, lst, lcv, idx, qs, ql, kl_new, one), T * 8.0 * h * e + state, 4.0 * T * h * e * e,
            like_bytes=T * (pxd.shape[1] * 2.0 + h * e * 8) + state, like_flops=9.0 * T * h * e * e, like_tflops=FP32_TFLOPS)
        wn, res = bf(h * e), bf(T, h * e)
        add("lightning_norm", "add_rms_norm", phase, lambda: L.lightning_norm(ro_o, gate, wn, h * e, h * e, 1e-6),
            lambda: ops.add_rms_norm(lo, res, wn, 1e-6, out=ro_o), T * h * e * 6.0, like_bytes=T * h * e * 8.0)
        lg, gl = torch.randn(B, s["vocab"], device="cuda"), bf(B, s["vocab"])
        add("softcap", "gelu_tanh", phase, lambda: ops.softcap(lg, 30.0), lambda: ops.gelu_tanh(gl), B * s["vocab"] * 8.0,
            like_bytes=B * s["vocab"] * 4.0)
        del kv, px, pxd, st, lst, gu, x, a, b, c, z
        torch.cuda.empty_cache()
    return rows


def main(sizes=tuple(SIZES), steps: int = 20) -> dict:
    return {"peaks": measured_peaks(), "fp32_tflops_nominal": FP32_TFLOPS, "kernels": [r for n in sizes for r in run_kernels(SIZES[n], n)],
            "models": list(run_models(sizes, steps=steps))}
