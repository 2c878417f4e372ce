"""Token-trace replay: given token ids go through a model step by step, and the logits asked for are written out.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps arrive on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

Every entry brings the next tokens of a request (admitted at its first entry) and the places among them whose logits
are wanted; all entries of a step run as one batch. ``end`` names requests to release after the step. A step with wanted
logits writes ``DIR/<step>.f32`` (little-endian fp32 [wanted, vocab], in the order of the entries); every step prints
``done <step>``.

The engine is the one that generates: architecture registry, weight loader, paged cache and state slots, batch packer
and the pipeline's step (:meth:`TextGenerationPipeline.score`), decode graphs included. Nothing is sampled. The cache pool
holds ``--max-tokens`` tokens in 64-token pages, and four requests may be live.
"""

from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np
import torch

from ..pipelines.context import TextContext

PAGE_TOKENS = 64
MAX_LIVE = 4


def build_engine(model_dir: str, dtype: torch.dtype, max_tokens: int, device: str):
    """An :class:`LLM` for a checkpoint directory with a cache pool of ``max_tokens`` tokens."""
    from ..pipelines.registry import PIPELINE_REGISTRY
    from ..pipelines.weights import load_hf_config, load_state_dict
    from .llm import LLM

    hf = load_hf_config(model_dir)
    arch = PIPELINE_REGISTRY.retrieve_architecture(hf)
    cfg = arch.config_class.from_hf(hf)
    weights = arch.weights_class.from_state_dict(cfg, load_state_dict(model_dir).to_dict(), torch.device(device), dtype)
    pages = -(-max_tokens // PAGE_TOKENS)
    tokens = pages * PAGE_TOKENS
    return LLM(cfg, weights, device=device, dtype=dtype, max_length=tokens, max_batch_size=MAX_LIVE,
               max_batch_input_tokens=tokens, page_size=PAGE_TOKENS, num_kv_pages=pages + 1, enable_prefix_caching=False,
               enable_overlap_scheduler=False, num_state_slots=MAX_LIVE, max_logit_rows=tokens)


class TraceSession:
    """Requests replayed through an engine's own step."""

    def __init__(self, llm):
        self.llm, self.live = llm, {}

    def step(self, entries: list, end: list) -> torch.Tensor:
        """Runs one batch; fp32 logits [wanted, vocab] of the wanted places, in the order of the entries."""
        kv, batch, want = self.llm.kv, [], []
        for e in entries:
            if not e["tokens"]:
                continue
            ctx = self.live.get(e["id"])
            if ctx is None:
                ctx = self.live[e["id"]] = TextContext.from_prompt(e["tokens"], self.llm.max_length, e["id"])
                kv.claim(ctx)
            else:
                ctx.tokens.extend(e["tokens"])
            kv.alloc(ctx)
            batch.append(ctx)
            want.append(e.get("want") or [])
        logits = self.llm.pipeline.score(batch, want) if batch else torch.empty(0, self.llm.cfg.vocab_size)
        for rid in end:
            if self.live.pop(rid, None) is not None:
                kv.release(rid)
        return logits


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a token trace and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32 files")
    ap.add_argument("--max-tokens", required=True, type=int, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default="cuda:0", help="cuda:N, or cpu for the PyTorch reference operations")
    args = ap.parse_args(argv)
    if args.device.startswith("cuda") and not torch.cuda.is_available():
        print("no CUDA device", file=sys.stderr)
        return 2
    session = TraceSession(build_engine(args.model, getattr(torch, args.dtype), args.max_tokens, args.device))
    for line in sys.stdin:
        if not line.strip():
            continue
        msg = json.loads(line)
        logits = session.step(msg.get("entries", []), msg.get("end", []))
        if any(e.get("want") for e in msg.get("entries", [])):
            data = logits.cpu().numpy().astype("<f4", copy=False)
            with open(os.path.join(args.out, f"{msg['step']}.f32"), "wb") as f:
                f.write(np.ascontiguousarray(data).tobytes())
        elif args.device.startswith("cuda"):
            torch.cuda.synchronize()
        print(f"done {msg['step']}", flush=True)
    if args.device.startswith("cuda"):
        from .. import ops

        ops.check_device_error()
    return 0
