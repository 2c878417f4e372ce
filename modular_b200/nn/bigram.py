"""Bigram embedding: every token adds a row chosen by itself and the token before it to its embedding.

The row is ``(previous * mul_prev + token * mul_cur) mod buckets``; a sequence's first token takes row ``buckets``. The previous
token of a step's first token lives in a state slot (``STATE``), so a step needs nothing but its own tokens; the rows are added
by the kernel that reads the embedding (:func:`modular_b200.nn.residual.sandwich_norm`, ``inject``).
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from .._native import lib as _lib

STATE = ("last_token", (1,), torch.int64)


@dataclass(frozen=True)
class BigramConfig:
    buckets: int
    mul_prev: int
    mul_cur: int

    def __post_init__(self):
        if self.buckets < 1 or self.mul_prev < 0 or self.mul_cur < 0:
            raise ValueError("a bigram table has at least one bucket, and multipliers are not negative")


def bigram_rows(cfg: BigramConfig, tokens, q_start, q_len, kv_len, state_idx, last):
    """Table rows int64 [T] of a ragged step; ``last`` [slots, 1] is read where a sequence continues, and advanced."""
    out = torch.empty_like(tokens)
    if tokens.is_cuda:
        _lib().bigram_rows(tokens, q_start, q_len, kv_len, state_idx, last, out, cfg.mul_prev, cfg.mul_cur, cfg.buckets)
        return out
    out.fill_(cfg.buckets)
    for s in range(q_len.numel()):
        t0, n, slot = int(q_start[s]), int(q_len[s]), int(state_idx[s])
        cur = tokens[t0: t0 + n]
        out[t0 + 1: t0 + n] = (cur[:-1] * cfg.mul_prev + cur[1:] * cfg.mul_cur) % cfg.buckets
        if slot >= 0 and n:
            if int(kv_len[s]) > n:
                out[t0] = (int(last[slot, 0]) * cfg.mul_prev + int(cur[0]) * cfg.mul_cur) % cfg.buckets
            last[slot, 0] = cur[-1]
    return out
