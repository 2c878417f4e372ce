"""Gotunex at sizes that resemble a real model's layers (random weights), beside the closest existing families.

``run_models``: prefill and decode throughput of whole models through the engine's step, Gotunex with a mix of latent and
delta-rule layers, Gotunex with latent layers only, and DeepSeek-V3 layers of the same width, heads, latents and experts.
``run_kernels``: every kernel of the design beside the like kernel of an existing family on the same shapes, with its
distance from a roofline (measured copy bandwidth, or the nominal fp32 rate for the recurrence).
"""

from __future__ import annotations

import torch

from .. import ops
from .._native import lib
from ..utils.peaks import measured_peaks
from .kernel_bench import time_fn

FP32_TFLOPS = 148 * 128 * 2 * 1.965e9 / 1e12        # nominal, CUDA cores
SIZES = {
    # width, layers, heads, dim, rot, vdim, kv_rank, q_rank, delta heads, delta dim, experts, top, expert ff, dense ff, vocab
    "w2048": dict(width=2048, layers=12, heads=16, dim=128, rot=64, vdim=128, kv_rank=512, q_rank=1536, dheads=16, ddim=128,
                  experts=64, top=6, expert_ff=1408, dense_ff=10944, vocab=102400),
    "w4096": dict(width=4096, layers=8, heads=32, dim=128, rot=64, vdim=128, kv_rank=512, q_rank=1536, dheads=32, ddim=128,
                  experts=32, top=4, expert_ff=2048, dense_ff=14336, vocab=128256),
    "w7168": dict(width=7168, layers=4, heads=128, dim=128, rot=64, vdim=128, kv_rank=512, q_rank=1536, dheads=64, ddim=128,
                  experts=32, top=4, expert_ff=2048, dense_ff=18432, vocab=129280),
}


def gotunex_config(s: dict, pattern: str):
    from ..models.gotunex import GotunexConfig

    att = dict(heads=s["heads"], dim=s["dim"], rot_dim=s["rot"], vdim=s["vdim"], kv_rank=s["kv_rank"], q_rank=s["q_rank"],
               scale=(s["dim"] + s["rot"]) ** -0.5, rot=dict(base=10000.0, dims=s["rot"]))
    delta = dict(heads=s["dheads"], kv_heads=s["dheads"], dim=s["ddim"], vdim=s["ddim"], conv=4)
    return GotunexConfig.build(s["width"], s["vocab"], pattern, att, delta, s["dense_ff"], s["expert_ff"], s["experts"], s["top"])


def deepseek_config(s: dict):
    from ..models.deepseek_v3 import DeepseekV3Config

    return DeepseekV3Config(vocab_size=s["vocab"], hidden_size=s["width"], intermediate_size=s["dense_ff"],
                            moe_intermediate_size=s["expert_ff"], num_hidden_layers=s["layers"], num_attention_heads=s["heads"],
                            q_lora_rank=s["q_rank"], kv_lora_rank=s["kv_rank"], qk_nope_head_dim=s["dim"],
                            qk_rope_head_dim=s["rot"], v_head_dim=s["vdim"], n_routed_experts=s["experts"], n_shared_experts=0,
                            num_experts_per_tok=s["top"], n_group=1, topk_group=1, first_k_dense_replace=1, rope_scaling=None,
                            max_position_embeddings=1 << 16)


def layer_pattern(n: int, delta: bool) -> str:
    """First layer with a dense feed-forward; with ``delta`` three recurrent layers per latent one and every second latent
    layer reading the one before."""
    if not delta:
        return "a" + "A" * (n - 1)
    out = "".join("DDDA"[i % 4] if (i // 4) % 2 == 0 else "DDDS"[i % 4] for i in range(n))
    return out[0].lower() + out[1:]


def bench_engine(cfg, prefill: int, seqs: int, batch: int, context: int, steps: int, seed: int = 0) -> dict:
    """Device times of prefill steps (``seqs`` prompts of ``prefill`` tokens) and of decode steps (``batch`` sequences with
    ``context`` tokens each, one graph replay per step), through the engine's own step."""
    import numpy as np

    from ..entrypoints.llm import LLM
    from ..models import family_for
    from ..pipelines.context import SamplingParams, TextContext

    n_tok = max(prefill * seqs, context * 4)
    page = 128
    need = max(seqs * (-(-prefill // page)), batch * (-(-(context + steps + 16) // page))) + 2
    fam = family_for(cfg)
    if hasattr(fam.weights_class, "random_init_ep"):       # generated on the device
        weights = fam.weights_class.random_init_ep(cfg, 0, 1, "cuda:0", torch.bfloat16, seed=seed, fp8_experts=False)
    else:
        weights = fam.weights_class.random_init(cfg, "cuda:0", torch.bfloat16, seed=seed)
    llm = LLM(cfg, weights, device="cuda:0", dtype=torch.bfloat16, max_length=max(prefill, context + steps + 16) + 128,
              max_batch_size=max(batch, seqs), max_batch_input_tokens=n_tok, page_size=page, num_kv_pages=need, enable_prefix_caching=False,
              enable_overlap_scheduler=False, graph_batch_sizes=[batch], seed=seed)
    native = llm.model.use_executor
    rng = np.random.default_rng(seed)
    ids = lambda n: rng.integers(0, cfg.vocab_size, size=n)
    n_ctx = 0

    def admit(n):
        nonlocal n_ctx
        n_ctx += 1
        c = TextContext.from_prompt(ids(n), llm.max_length, f"r{n_ctx}", SamplingParams(temperature=0.0, ignore_eos=True))
        llm.kv.claim(c)
        llm.kv.alloc(c)
        return c

    def timed(ctxs, want):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        if native:                       # the step runs in the native executor and samples greedily
            llm.pipeline.execute(ctxs)
        else:
            llm.pipeline.score(ctxs, want)
        b.record()
        b.synchronize()
        return a.elapsed_time(b)

    pre = []
    for _ in range(3 + 5):
        ctxs = [admit(prefill) for _ in range(seqs)]
        pre.append(timed(ctxs, [[prefill - 1]] * seqs))
        for c in ctxs:
            llm.kv.release(c.request_id)
    ctxs = []
    while len(ctxs) < batch:
        part = [admit(context) for _ in range(min(4, batch - len(ctxs)))]
        timed(part, [[]] * len(part))
        ctxs += part
    dec = []
    for _ in range(5 + steps):
        for c in ctxs:
            if not native:
                c.tokens.extend(ids(1))
            llm.kv.alloc(c)
        dec.append(timed(ctxs, [[0]] * batch))
    ops.check_device_error()
    med = lambda v: sorted(v)[len(v) // 2]
    p, d = med(pre[3:]), med(dec[5:])
    return {"params": cfg.param_count(), "prefill_tokens": prefill * seqs, "prefill_ms": p, "prefill_tok_s": prefill * seqs / p * 1e3,
            "decode_batch": batch, "context": context, "decode_ms": d, "decode_tok_s": batch / d * 1e3,
            "graph_replays": getattr(llm.model, "graph_replays", None)}


def run_models(sizes=("w2048", "w4096", "w7168"), prefill=2048, seqs=4, batches=(1, 64), context=2048, steps=20):
    """Yields one record per (size, model, decode batch)."""
    import gc

    for name in sizes:
        s = SIZES[name]
        for label, cfg in (("gotunex (delta + latent)", gotunex_config(s, layer_pattern(s["layers"], True))),
                           ("gotunex (latent only)", gotunex_config(s, layer_pattern(s["layers"], False))),
                           ("deepseek-v3 layers", deepseek_config(s))):
            for batch in batches:
                r = bench_engine(cfg, prefill, seqs, batch, context, steps)
                yield {"size": name, "model": label, "layers": s["layers"], **r}
                gc.collect()
                torch.cuda.empty_cache()


def _cache(B: int, context: int, width: int, page: int = 128):
    """(cache [pages, page, width], block table [B, n]) of ``B`` sequences."""
    n = -(-context // page)
    cache = torch.randn(B * n, page, width, device="cuda").bfloat16()
    return cache, torch.randperm(B * n, device="cuda").int().view(B, n)


def run_kernels(s: dict, name: str, prefill: int = 2048, seqs: int = 4, batch: int = 64, context: int = 2048) -> list:
    """Every kernel of the design beside the like kernel of an existing family, same shapes, L2 flushed."""
    from ..nn import state_space
    from ..nn.delta_rule import DeltaRule, DeltaRuleConfig, delta_rule_cuda
    from ..nn.latent_attention import latent_attention, rotate_heads
    from ..nn.moe import TableRouter
    from ..nn.residual import residual_norm
    from ..nn.rotary_embedding import cos_sin_table

    peaks, rows, L = measured_peaks(), [], lib()
    bf = lambda *shape: torch.randn(*shape, device="cuda").bfloat16()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    W, H, R, D, d, vd = s["width"], s["heads"], s["kv_rank"], s["rot"], s["dim"], s["vdim"]

    def add(kernel, like, phase, fn, like_fn, nbytes, flops=0.0, peak_tflops=None, like_bytes=None, like_flops=None):
        t = time_fn(fn)
        roof = lambda b, f: max(b / (peaks["hbm_gbs"] * 1e9), f / ((peak_tflops or peaks["bf16_tflops"]) * 1e12))
        r = {"size": name, "kernel": kernel, "phase": phase, "us": t * 1e6, "frac_of_roofline": roof(nbytes, flops) / t, "like": like}
        if like_fn is not None:
            u = time_fn(like_fn)
            r.update(like_us=u * 1e6, like_frac=roof(nbytes if like_bytes is None else like_bytes,
                                                     flops if like_flops is None else like_flops) / u)
        rows.append(r)

    for phase, T, B, ctx in (("prefill", prefill * seqs, seqs, prefill), ("decode", batch, batch, context), ("decode b1", 1, 1, context)):
        one = T == B
        ql, kl = i32([T // B] * B), i32([ctx] * B)
        qs = (torch.cumsum(ql, 0) - ql).int()
        pos = torch.arange(T, device="cuda", dtype=torch.int32) % ctx
        # --- latent attention, with a sink, beside the same attention without one
        cache, bt = _cache(B, ctx, R + D)
        slots = (bt.repeat_interleave(T // B, 0)[torch.arange(T, device="cuda"), pos.long() // 128].long() * 128 + pos.long() % 128)
        q_lat, q_rope, sink = bf(T, H, R), bf(T, H, D), torch.randn(H, device="cuda")
        pairs = B * ctx if one else B * ctx * (ctx + 1) // 2
        fl = 2.0 * pairs * H * (2 * R + D)
        by = 2.0 * (T * H * (2 * R + D) + B * ctx * (R + D))
        add("latent attention (sink)", "mla_paged_attention", phase,
            lambda: latent_attention(q_lat, q_rope, cache, bt, qs, ql, kl, 0.1, sink, one),
            lambda: ops.mla_paged_attention(q_lat, q_rope, cache, bt, qs, ql, kl, 0.1), by, fl)
        # --- after the down-projections, and the query rotation
        px, g1, g2, cs = bf(T, s["q_rank"] + R + D + H * vd), bf(s["q_rank"]), bf(R), cos_sin_table(D, ctx + 1, 1e4, None, "cuda")
        cq = torch.empty(T, s["q_rank"], device="cuda", dtype=torch.bfloat16)
        by = 2.0 * T * 2 * (s["q_rank"] + R + D)
        add("latent_post_down", "mla_post_down", phase,
            lambda: L.latent_post_down(px, s["q_rank"], g1, cq, s["q_rank"], R, R, g2, D, D, D, False, 1e-6, pos, cs, slots, cache),
            lambda: L.mla_post_down(px, s["q_rank"], g1, g2, 1e-6, pos, cs, slots, cq, cache), by)
        q = bf(T, H * (d + D))
        add("rotate_heads", "mla_q_rope", phase, lambda: rotate_heads(q[:, d:], H, d + D, D, False, pos, cs),
            lambda: L.mla_q_rope(q, H, d, pos, cs, q_rope), 4.0 * T * H * D)
        o = bf(T, H * vd)
        gu = bf(T, 2 * H * vd)
        add("sigmoid_gate", "silu_mul", phase, lambda: ops.sigmoid_gate(o, px[:, s["q_rank"] + R + D:], H * vd),
            lambda: ops.silu_mul(gu, o), 6.0 * T * H * vd)
        u, gu2 = bf(T, s["dense_ff"]), bf(T, 2 * s["dense_ff"])
        uo = torch.empty_like(u)
        add("gelu_tanh", "silu_mul", phase, lambda: ops.gelu_tanh(u), lambda: ops.silu_mul(gu2, uo), 4.0 * T * s["dense_ff"],
            like_bytes=6.0 * T * s["dense_ff"])
        # --- residual seam: both branches and both norms; the like kernel adds one branch and writes one norm
        x, a, b, w1, w2, n1, n2 = torch.randn(T, W, device="cuda"), bf(T, W), bf(T, W), bf(W), bf(W), bf(T, W), bf(T, W)
        add("residual_norm", "add_rmsnorm", phase, lambda: residual_norm(x, a=a, b=b, w1=w1, n1=n1, w2=w2, n2=n2),
            lambda: ops.add_rms_norm(a, b, w1, 1e-6, out=n1), T * W * (8.0 + 4.0 + 4.0), like_bytes=T * W * 8.0)
        # --- expert order of every layer at once, and the seam that reads and writes it, beside sort + permute + combine
        E, k, n_moe = s["experts"], s["top"], s["layers"] - 1
        V = 4096
        tab = [torch.rand(V, E).topk(k, -1).indices.int() for _ in range(n_moe)]
        router, ids = TableRouter(tab, [E] * n_moe, "cuda"), torch.randint(0, V, (T,), device="cuda")
        inv, _ = router.route(ids)[0]
        eo, n2s = bf(T * k, W), bf(T * k, W)
        top = router.tables[0][ids].contiguous()
        wts = torch.full((T, k), 1.0 / k, device="cuda")
        scratch, offs = torch.zeros(2 * E, dtype=torch.int32, device="cuda"), torch.empty(E + 1, dtype=torch.int32, device="cuda")
        order, inverse = (torch.empty(T * k, dtype=torch.int32, device="cuda") for _ in range(2))

        def like_sort():
            for _ in range(n_moe):
                L.moe_create_indices(top, 0, E, scratch, offs, order, inverse)

        add(f"moe_table_route ({n_moe} layers)", f"moe_create_indices x {n_moe}", phase, lambda: router.route(ids), like_sort,
            n_moe * T * (8.0 + 8.0 * k))
        like_sort()

        def like_moe():
            L.moe_combine(eo, inverse, wts, None, n1, k)
            ops.add_rms_norm(a, b, w1, 1e-6, out=n1)
            L.moe_permute_rows(n1, order, offs[E:], n2s, k)

        add("residual_norm (experts)", "combine + add_rmsnorm + permute", phase,
            lambda: residual_norm(x, a=a, e=eo, inverse=inv, pair_w=1 / k, w1=w1, n1=n1, w2=w2, n2=n2s, scatter=inv), like_moe,
            T * W * (8.0 + 4.0 + 4.0 * k), like_bytes=T * W * (8.0 + 4.0 * k + 4.0))
        # --- recurrence: the same state size as the SSD scan of state-space layers
        dh, dd = s["dheads"], s["ddim"]
        c = DeltaRuleConfig(W, dh, dh, dd, dd, 4, dd, dd, 1e-6)
        m = DeltaRule.__new__(DeltaRule)
        m.cfg, m.off = c, {n: at for n, _, at in c.blocks}
        last = c.blocks[-1]
        pxd = bf(T, last[2] + last[1])
        m.conv_w, m.A_log, m.dt_bias, m.norm = bf(c.channels, 4), torch.zeros(dh, device="cuda"), torch.zeros(dh * dd, device="cuda"), bf(dd)
        z, gate, out = torch.randn(T, dh * dd, device="cuda"), bf(T, dh * dd), bf(T, dh * dd)
        st, cv = (torch.zeros(B, *sh, device="cuda") for sh in (c.state_shapes()["delta"], c.state_shapes()["conv"]))
        idx = torch.arange(B, device="cuda", dtype=torch.int32)
        kl_new = ql if not one else kl
        state_bytes = B * dh * dd * dd * 4.0 * (2 if one else 1)
        by = T * (pxd.shape[1] * 2.0 + dh * dd * (4 + 2 + 2)) + state_bytes
        fl = 9.0 * T * dh * dd * dd               # decay, two products of 2, update of 2, per state element
        xs, dts, Bm = bf(T, dh, dd), bf(T, dh), bf(T, 1, dd)
        A, Dk, dtb = -torch.ones(dh, device="cuda"), torch.ones(dh, device="cuda"), torch.zeros(dh, device="cuda")
        cu = torch.cat([qs, i32([T])]).int()
        init = (kl_new > ql).int()
        like_fl = 5.0 * T * dh * dd * dd
        add("delta rule", "ssd_scan_varlen", phase,
            lambda: delta_rule_cuda(m, pxd, z, gate, out, st, cv, idx, qs, ql, kl_new, one),
            lambda: state_space.ssd_scan_varlen(xs, dts, A, Bm, Bm, Dk, dtb, cu, st, idx, init), by, fl, FP32_TFLOPS,
            like_bytes=T * dh * dd * 4.0 + state_bytes, like_flops=like_fl)
        del cache, q_lat, q_rope, px, eo, n2s, pxd, st
        torch.cuda.empty_cache()
    return rows


def main(sizes=("w2048", "w4096", "w7168"), steps: int = 20) -> dict:
    return {"peaks": measured_peaks(), "fp32_tflops_nominal": FP32_TFLOPS, "models": list(run_models(sizes, steps=steps)),
            "kernels": [r for n in sizes for r in run_kernels(SIZES[n], n)]}
