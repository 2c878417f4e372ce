"""The seam between two layers of a decoder whose residual stream is kept in fp32.

``residual_norm`` adds what the branches of the last layer produced and writes the normalised input of every branch of
the next one in a single kernel (``csrc/kernels/residual_norm.cu``); the PyTorch form below runs on CPU tensors.

* ``table`` / ``ids`` / ``scale``: the stream starts as scaled embedding rows instead of what ``x`` holds;
* ``a``, ``b``: branch outputs; ``e`` with ``inverse`` [T, k] and ``pair_w``: expert outputs in expert order, summed per
  token (a mixture-of-experts branch without a combine kernel);
* ``w1``/``n1`` and ``w2``/``n2``: norm weights and outputs of up to two parallel branches; ``scatter`` [T, k] writes
  the second one to the rows a token occupies in expert order (no permute kernel);
* ``norm_a`` / ``norm_b``: the branches ``a`` and ``b`` are RMS-normed with these weights before they are added;
  ``ab_scale`` multiplies them, ``c`` is a third branch (no norm), ``mult`` multiplies the whole update;
* ``inject``: adds ``inject_scale * inject[ids]`` to the stream, ``step`` one row to every token (what a looped pass adds
  before its first layer);
* ``rows``: work on these rows of ``x`` only (the ones whose logits are wanted), outputs compacted.

``sandwich_norm`` is the seam of layers that norm every branch before *and* after it, one branch at a time:
``x += mult * norm(u; w_u, b_u)`` with ``u`` a branch output or the weighted sum of expert outputs in expert order, then
``n1 = norm(x; w1, b1)``; layer norms with biases, RMS norms without. ``inject`` adds rows of a second table, chosen by ids of
their own, to the embedding.

``tanh_seam`` (``csrc/kernels/tanh_seam.cu``) is the same seam for elementwise norms, dynamic tanh ``T(y) = tanh(alpha * y) * w + b``,
each given as a triple ``(alpha, w, b)``: ``x_out = x + T(u)``, ``n1 = T(x_out)``. The branch ``u`` is ``a``, the weighted expert
outputs ``e``, or their sum; a pair whose ``inverse`` is negative belongs to an identity expert and gives the token's row of
``self_rows``. With a ``shift`` vector, ``n1[t]`` moves by it towards the normed row of the token before. That needs a second buffer
``x_out`` and the sequences of the step; ``prev`` [slots, width] keeps every sequence's last normed row.

The norm is computed in fp32 and rounded once.
"""

from __future__ import annotations

import torch

from .._native import lib as _lib


def residual_norm_reference(x, ids=None, table=None, scale=1.0, a=None, b=None, e=None, inverse=None, pair_w=1.0, rows=None,
                            w1=None, n1=None, w2=None, n2=None, scatter=None, cols=0, store_x=True, eps=1e-6,
                            norm_a=None, norm_b=None, ab_scale=1.0, c=None, mult=1.0, inject=None, inject_scale=1.0, step=None):
    cols = cols or x.shape[1]
    idx = torch.arange(x.shape[0]) if rows is None else rows.long()
    h = x[idx] if table is None else table[ids[idx]].float() * scale
    s = torch.zeros_like(h)

    def branch(t, w):
        y = t[idx, : x.shape[1]].float()
        return y if w is None else y * torch.rsqrt((y * y).sum(-1, keepdim=True) / cols + eps) * w.float()

    if e is not None:
        inv = inverse.view(x.shape[0], -1)[idx].long()
        got = e[inv.clamp(min=0)].float() * (inv >= 0).unsqueeze(-1)
        s = got.sum(1) * pair_w
    elif b is not None:
        s = branch(b, norm_b)
    if a is not None:
        s = s + branch(a, norm_a)
    s = s * ab_scale
    if c is not None:
        s = s + branch(c, None)
    h = h + s * mult
    if inject is not None:
        h = h + inject[ids[idx]].float() * inject_scale
    if step is not None:
        h = h + step.float()
    if store_x:
        x[idx] = h
    if w1 is None:
        return
    n = h * torch.rsqrt((h * h).sum(-1, keepdim=True) / cols + eps)
    n1[: idx.numel()] = (n * w1.float()).to(n1.dtype)
    if w2 is not None:
        y = (n * w2.float()).to(n2.dtype)
        if scatter is None:
            n2[: idx.numel()] = y
        else:
            for k in range(scatter.shape[1]):
                pos = scatter[idx, k].long()
                n2[pos[pos >= 0]] = y[pos >= 0]


def residual_norm(x, ids=None, table=None, scale=1.0, a=None, b=None, e=None, inverse=None, pair_w=1.0, rows=None, w1=None,
                  n1=None, w2=None, n2=None, scatter=None, cols=0, store_x=True, eps=1e-6, norm_a=None, norm_b=None, ab_scale=1.0, c=None, mult=1.0,
                  inject=None, inject_scale=1.0, step=None):
    """x: fp32 [T, width], width padded to a multiple of 4 with zeros; ``cols`` is the true width (the norm's divisor)."""
    if not x.is_cuda:
        return residual_norm_reference(x, ids, table, scale, a, b, e, inverse, pair_w, rows, w1, n1, w2, n2, scatter, cols,
                                       store_x, eps, norm_a, norm_b, ab_scale, c, mult, inject, inject_scale, step)
    _lib().residual_norm(x, ids, table, float(scale), a, b, e, inverse, 0 if inverse is None else inverse.numel() // x.shape[0],
                         float(pair_w), rows, w1, n1, w2, n2, scatter, cols or x.shape[1], store_x, float(eps),
                         x.shape[0] if rows is None else rows.numel(), norm_a, norm_b, float(ab_scale), c, float(mult), inject,
                         float(inject_scale), step)


def sandwich_norm_reference(x, ids=None, table=None, scale=1.0, inject_ids=None, inject=None, a=None, e=None, inverse=None, pair_w=None,
                            rows=None, w_u=None, b_u=None, mult=1.0, w1=None, b1=None, n1=None, cols=0, store_x=True, eps=1e-6):
    cols = cols or x.shape[1]
    idx = torch.arange(x.shape[0]) if rows is None else rows.long()

    def norm(t, w, b):
        d = t[:, :cols]
        if b is not None:
            d = d - d.mean(-1, keepdim=True)
        y = torch.zeros_like(t)
        y[:, :cols] = d * torch.rsqrt((d * d).mean(-1, keepdim=True) + eps) * w.float()[:cols]
        if b is not None:
            y[:, :cols] += b.float()[:cols]
        return y

    h = x[idx] if table is None else table[ids[idx]].float() * scale
    if inject is not None:
        h = h + inject[inject_ids[idx]].float()
    u = None
    if a is not None:
        u = a[idx, : x.shape[1]].float()
    elif e is not None:
        inv = inverse[idx].long()
        u = (e[inv.clamp(min=0)].float() * (pair_w[idx] * (inv >= 0)).unsqueeze(-1)).sum(1)
    if u is not None:
        h = h + mult * (u if w_u is None else norm(u, w_u, b_u))
    if store_x:
        x[idx] = h
    if w1 is not None:
        n1[: idx.numel()] = norm(h, w1, b1).to(n1.dtype)


def sandwich_norm(x, ids=None, table=None, scale=1.0, inject_ids=None, inject=None, a=None, e=None, inverse=None, pair_w=None, rows=None,
                  w_u=None, b_u=None, mult=1.0, w1=None, b1=None, n1=None, cols=0, store_x=True, eps=1e-6):
    """x: fp32 [T, width], width padded to a multiple of 4 with zeros; ``cols`` is the true width."""
    if not x.is_cuda:
        return sandwich_norm_reference(x, ids, table, scale, inject_ids, inject, a, e, inverse, pair_w, rows, w_u, b_u, mult, w1, b1, n1,
                                       cols, store_x, eps)
    _lib().sandwich_norm(x, ids, table, float(scale), inject_ids, inject, a, e, inverse, pair_w, rows, w_u, b_u, float(mult), w1, b1, n1,
                         cols or x.shape[1], store_x, float(eps), x.shape[0] if rows is None else rows.numel())


def tanh_seam_reference(x=None, x_out=None, ids=None, table=None, scale=1.0, a=None, e=None, inverse=None, pair_w=None, self_rows=None,
                        rows=None, norm_u=None, norm1=None, n1=None, shift=None, prev=None, state_idx=None, q_start=None, q_len=None,
                        kv_len=None):
    T = lambda y, n: torch.tanh(n[0] * y) * n[1].float() + n[2].float()
    idx = torch.arange(x.shape[0] if x is not None else ids.numel()) if rows is None else rows.long()
    h = x[idx] if table is None else table[ids[idx]].float() * scale
    u = None if a is None else a[idx, : h.shape[1]].float()
    if e is not None:
        inv, w = inverse[idx].long(), pair_w[idx].unsqueeze(-1)
        y = torch.where((inv >= 0).unsqueeze(-1), e[inv.clamp(min=0)].float(), 0.0)
        if self_rows is not None:
            y = torch.where((inv >= 0).unsqueeze(-1), y, self_rows[idx, : h.shape[1]].float().unsqueeze(1))
        u = (y * w).sum(1) if u is None else u + (y * w).sum(1)
    if u is not None:
        h = h + T(u, norm_u)
    if x_out is not None:
        x_out[idx] = h
    if norm1 is None:
        return
    y = T(h, norm1)
    if shift is not None:
        before = torch.zeros_like(y)
        before[1:] = y[:-1]
        for s in range(q_len.numel()):
            t0, n, slot = int(q_start[s]), int(q_len[s]), int(state_idx[s])
            if n == 0:
                continue
            before[t0] = prev[slot] if slot >= 0 and int(kv_len[s]) > n else 0.0
            if slot >= 0:
                prev[slot] = y[t0 + n - 1]
        y = y + (before - y) * shift.float()
    n1[: idx.numel()] = y.to(n1.dtype)


def tanh_seam(x=None, x_out=None, ids=None, table=None, scale=1.0, a=None, e=None, inverse=None, pair_w=None, self_rows=None, rows=None,
              norm_u=None, norm1=None, n1=None, shift=None, prev=None, state_idx=None, q_start=None, q_len=None, kv_len=None):
    """``x`` (or ``table`` rows) fp32 [T, width] -> ``x_out`` (may be ``x`` without a shift; None: not stored) and ``n1``."""
    some = x if x is not None else table
    if not some.is_cuda:
        return tanh_seam_reference(x, x_out, ids, table, scale, a, e, inverse, pair_w, self_rows, rows, norm_u, norm1, n1, shift, prev,
                                   state_idx, q_start, q_len, kv_len)
    if e is None:
        self_rows = None
    n_rows = rows.numel() if rows is not None else x.shape[0] if x is not None else ids.numel()
    (au, wu, bu), (a1, w1, b1) = norm_u or (0.0, None, None), norm1 or (0.0, None, None)
    _lib().tanh_seam(x, x_out, ids, table, float(scale), a, e, inverse, pair_w, self_rows, rows, wu, bu, au, w1, b1, a1, n1, shift, prev,
                     state_idx, q_start, q_len, kv_len, shift is not None and n_rows == q_len.numel(), some.shape[1], n_rows)
