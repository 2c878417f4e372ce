"""CUDA graphs of decode steps for models whose step is driven op by op from Python.

A graph covers one batch size with one token per sequence. A step of fewer sequences replays the next larger graph with
dummy sequences on the null page (slot -1: they store nothing in the cache, nothing in a recurrent state).
"""

from __future__ import annotations

import contextlib
import gc
from typing import Sequence

import torch


@contextlib.contextmanager
def no_gc_during_capture():
    """Collect dead reference cycles now and keep the cyclic collector off while a CUDA graph is captured. The
    step runs as Python code that allocates many temporaries; a collection triggered in the middle of it
    can destroy CUDA graphs of an engine that is no longer referenced, and destroying a graph is not permitted
    while a stream captures (the capture is invalidated and the next launch fails)."""
    gc.collect()
    was_on = gc.isenabled()
    gc.disable()
    try:
        yield
    finally:
        if was_on:
            gc.enable()


class DecodeGraphs:
    """``step(**tensors) -> logits`` captured once per batch size over static input tensors."""

    FIELDS = (("tokens", torch.int64, 0), ("positions", torch.int32, 0), ("slots", torch.int64, -1),
              ("kv_len", torch.int32, 1), ("state_slot", torch.int32, -1))

    def __init__(self, step, device, max_pages: int, max_seqs: int):
        self.step, self.device, self.max_pages, self.max_seqs = step, device, max_pages, max_seqs
        self.graphs: dict = {}
        self.replays = 0
        self.replayed_calls = 0          # native calls inside replayed graphs (0 unless calls are counted)

    def capture(self, batch_sizes: Sequence[int]) -> None:
        from .._native import native_calls

        dev = self.device
        for B in sorted(set(int(b) for b in batch_sizes)):
            if B in self.graphs or B > self.max_seqs:
                continue
            st = {n: torch.full((B,), fill, dtype=dt, device=dev) for n, dt, fill in self.FIELDS}
            ar = torch.arange(B, dtype=torch.int32, device=dev)
            st.update(block_table=torch.zeros(B, self.max_pages, dtype=torch.int32, device=dev), q_start=ar,
                      q_len=torch.ones_like(ar), logit_rows=ar.clone())
            side = torch.cuda.Stream(device=dev)
            side.wait_stream(torch.cuda.current_stream())
            with torch.cuda.stream(side):
                self.step(**st)
            torch.cuda.current_stream().wait_stream(side)
            torch.cuda.synchronize()
            g, n0 = torch.cuda.CUDAGraph(), native_calls()
            with no_gc_during_capture():
                with torch.cuda.graph(g):
                    logits = self.step(**st)
            self.graphs[B] = (g, st, logits, native_calls() - n0)
        torch.cuda.synchronize()

    def fits(self, T: int, n_seqs: int, n_logits: int) -> int:
        """The graph size for a step, or 0."""
        if not self.graphs or not T == n_seqs == n_logits:
            return 0
        return min((b for b in self.graphs if b >= T), default=0)

    def replay(self, size: int, block_table: torch.Tensor, **tensors) -> torch.Tensor:
        g, st, logits, calls = self.graphs[size]
        n = tensors["tokens"].shape[0]
        for name, _, fill in self.FIELDS:
            if tensors.get(name) is not None:
                st[name][:n].copy_(tensors[name])
            if n < size:
                st[name][n:].fill_(fill)
        w = min(block_table.shape[1], self.max_pages)
        st["block_table"][:n, :w].copy_(block_table[:, :w])
        g.replay()
        self.replays += 1
        self.replayed_calls += calls
        return logits[:n]
