"""Softmax attention and a gated delta rule side by side: both read one input, and the layer's output is their scaled sum.

The projections of both are one stacked GEMM, and so are the output projections: the attention kernel and the delta rule write
their heads, already gated and scaled, next to each other, and one product over all of them gives the sum.
"""

from __future__ import annotations

import torch
import torch.nn.functional as F

from .delta_rule import DeltaRule, gemm_k
from .window_attention import WindowAttention


class ParallelMixer:
    """``left`` with a head gate and ``right`` carry their factors (``out_mult``) in their configs."""

    def __init__(self, left: WindowAttention, right: DeltaRule, device, dtype):
        self.left, self.right = left, right
        self.w_in = torch.cat([left.w_in.to(device=device, dtype=dtype), right.w_in]).contiguous()
        self.left_cols, self.right_cols = left.w_o.shape[1], right.cfg.heads * right.cfg.vdim
        self.w_o = torch.cat([left.w_o, right.w_o[:, : self.right_cols]], 1)
        self.w_o = F.pad(self.w_o, (0, gemm_k(self.w_o.shape[1]) - self.w_o.shape[1])).contiguous()
        left.w_in = right.w_in = left.w_o = right.w_o = None        # the stacked copies are the ones in use

    def __call__(self, x, lin, kv, plane: int, state, conv_state, cos_sin, positions, slots, block_table, q_start, q_len, kv_len, state_idx,
                 plan, one_token: bool):
        """x [T, width] -> [T, width]."""
        left, right, T = self.left, self.right, x.shape[0]
        px = lin(x, self.w_in)
        left.prep(px, positions, cos_sin, slots, kv, plane)
        heads = torch.empty(T, self.w_o.shape[1], dtype=x.dtype, device=x.device)
        end = self.left_cols + self.right_cols
        if heads.shape[1] != end:
            heads[:, end:].zero_()
        left(px[:, : left.k_off], kv, plane, block_table, q_start, q_len, kv_len, plan, heads[:, : self.left_cols],
             px[:, left.g_off: left.g_off + left.cfg.heads_pad])
        right.mix(px[:, left.in_rows:], heads[:, self.left_cols:], state, conv_state, state_idx, q_start, q_len, kv_len, one_token)
        return lin(heads, self.w_o)
