"""A block whose branches all read one normalised input: windowed softmax attention, lightning attention and a squared-relu
feed-forward side by side.

Every projection of the input is one stacked GEMM (attention q, k, v; lightning q, k, v, gate; feed-forward up), and one
kernel (:func:`modular_b200.nn.window_attention.block_prep`) does everything between it and the branches. The block returns
its branch outputs; the seam of the next layer (:func:`modular_b200.nn.residual.residual_norm`) norms, averages and adds them.
"""

from __future__ import annotations

from typing import Optional

import torch
import torch.nn.functional as F

from .delta_rule import gemm_k, pad_to
from .lightning_attention import LightningAttention
from .window_attention import WindowAttention, block_prep


class ParallelBlock:
    def __init__(self, left: WindowAttention, right: LightningAttention, norm_left, norm_right, up: Optional[torch.Tensor],
                 down: Optional[torch.Tensor], width_pad: int, device, dtype):
        put = lambda t: t.to(device=device, dtype=dtype).contiguous()
        row = lambda t: put(F.pad(t, (0, width_pad - t.shape[0])))
        self.left, self.right = left, right
        self.norm_left, self.norm_right = row(norm_left), row(norm_right)
        self.right_off = left.in_rows
        self.up_off = self.right_off + right.in_rows
        parts, self.ff, self.w_down = [left.w_in, right.w_in], 0, None
        if up is not None:
            self.ff = gemm_k(up.shape[0])
            parts.append(pad_to(up, self.ff, width_pad))
            self.w_down = put(pad_to(down, width_pad, self.ff))
        self.w_in = put(torch.cat(parts))
        left.w_in = right.w_in = None                       # the stacked copy is the one in use

    def __call__(self, h, lin, kv, plane, state, cos_sin, positions, slots, block_table, q_start, q_len, kv_len, state_idx, plan,
                 one_token: bool) -> dict:
        """h [T, width] -> the branch outputs as arguments of ``residual_norm``."""
        left, right = self.left, self.right
        px = lin(h, self.w_in)
        block_prep(px, left.cfg.heads_pad, left.k_off, left.v_off, left.cfg.kv_heads, left.cfg.rot_dims, positions, cos_sin, slots, kv,
                   plane, silu=(self.right_off, right.act_rows), relu2=(self.up_off, self.ff))
        a = left(px[:, : left.k_off], kv, plane, block_table, q_start, q_len, kv_len, plan)
        b = right(px[:, self.right_off: self.up_off], state, state_idx, q_start, q_len, kv_len, one_token)
        out = dict(a=lin(a, left.w_o), b=lin(b, right.w_o), norm_a=self.norm_left, norm_b=self.norm_right, ab_scale=0.5)
        if self.w_down is not None:
            out["c"] = lin(px[:, self.up_off: self.up_off + self.ff], self.w_down)
        return out
