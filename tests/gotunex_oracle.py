"""Plain implementation of the Gotunex design for tests: one function per mechanism, one sequence at a time, no cache,
no batching, no code shared with the package. ``cfg`` is the parsed config.json, ``w`` a dict of tensors by name.
Everything runs in the dtype of ``DT`` (float64 by default)."""

import math

import torch

DT = torch.float64


def rms(x, weight, eps):
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(x, dims, base, first_position=0):
    """x [T, heads, d]: the first ``dims`` values of every head rotate, value i together with value i + dims / 2."""
    T = x.shape[0]
    half = dims // 2
    out = x.clone()
    for p in range(T):
        for i in range(half):
            a = (first_position + p) * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            u, v = x[p, :, i], x[p, :, i + half]
            out[p, :, i] = u * c - v * s
            out[p, :, i + half] = v * c + u * s
    return out


def short_conv(x, taps):
    """x [T, C], taps [C, n]: the last column of ``taps`` meets the current token; silu after it."""
    T, n = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(n):
            src = t - (n - 1) + j
            if src >= 0:
                out[t] += taps[:, j] * x[src]
    return silu(out)


def latent_rows(h, w, p, m, eps):
    """What a layer with its own W_dkv keeps per token: (latent [T, kv_rank], rotated key part [T, rot_dim])."""
    a = h @ w[p + "dkv"].T
    c = rms(a[:, : m["kv_rank"]], w[p + "dkv.norm"], eps)
    kr = rotate(a[:, m["kv_rank"]:].unsqueeze(1), m["rot"]["dims"], m["rot"]["base"])[:, 0]
    return c, kr


def latent_attention(h, w, p, m, eps, rows):
    T, H, d, r, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = rows
    q = (rms(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).view(T, H, d + r)
    qn, qr = q[..., :d], rotate(q[..., d:], m["rot"]["dims"], m["rot"]["base"])
    k = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    visible = torch.ones(T, T, dtype=torch.bool).tril()
    for i in range(H):
        s = (qn[:, i] @ k[:, i].T + qr[:, i] @ kr.T) * m["scale"]
        s = torch.where(visible, s, torch.full_like(s, -math.inf))
        sink = w[p + "sink"][i]
        top = torch.maximum(s.max(dim=1, keepdim=True).values, sink)
        e = torch.exp(s - top)
        out[:, i] = (e / (e.sum(dim=1, keepdim=True) + torch.exp(sink - top))) @ v[:, i]
    return (out.reshape(T, H * dv) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def delta_recurrence(q, k, v, g, beta, state):
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H], state [H, d, dv]: outputs [T, H, dv] and the state after."""
    out = []
    for t in range(q.shape[0]):
        state = state * g[t].unsqueeze(-1)
        u = beta[t].unsqueeze(-1) * (v[t] - torch.einsum("hdv,hd->hv", state, k[t]))
        state = state + k[t].unsqueeze(-1) * u.unsqueeze(1)
        out.append(torch.einsum("hdv,hd->hv", state, q[t]))
    return torch.stack(out), state


def channel_delta(h, w, p, m, eps):
    T, H, KH, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ w[p + "q"].T, w[p + "q.conv"]).view(T, KH, d)
    k = short_conv(h @ w[p + "k"].T, w[p + "k.conv"]).view(T, KH, d)
    v = short_conv(h @ w[p + "v"].T, w[p + "v.conv"]).view(T, H, dv)
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    head_of = [i // (H // KH) for i in range(H)]
    q, k = (unit(q) / math.sqrt(d))[:, head_of], unit(k)[:, head_of]
    beta = sigmoid(h @ w[p + "b"].T)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    softplus = torch.where(z > 0, z + torch.log1p(torch.exp(-z.abs())), torch.log1p(torch.exp(-z.abs())))
    g = torch.exp(-torch.exp(w[p + "A_log"]).view(1, H, 1) * softplus.view(T, H, d))
    o, _ = delta_recurrence(q, k, v, g, beta, torch.zeros(H, d, dv, dtype=h.dtype))
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(T, H, dv)
    return (rms(o, w[p + "norm"], eps) * gate).reshape(T, H * dv) @ w[p + "o"].T


def dense_ff(h, w, p):
    return gelu_tanh(h @ w[p + "up"].T) @ w[p + "down"].T


def table_moe(h, tokens, w, p, top):
    table = w[p + "table"].long()
    out = torch.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in table[tok].tolist():
            q = f"{p}e{e}."
            out[t] += (w[q + "down"] @ (silu(w[q + "gate"] @ h[t]) * (w[q + "up"] @ h[t]))) / top
    return out


def forward(cfg, w, tokens):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    w = {k: (v if v.dtype in (torch.int32, torch.int64) else v.to(DT)) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    tokens = [int(t) for t in tokens]
    x = w["embed"][tokens] * cfg["embedding"]["scale"]
    kept, stream = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        n1 = rms(x, w[p + "norm1"], eps)
        if layer["type"] == "latent_attention":
            j = m.get("kv_from")
            if j is None:
                kept[i] = latent_rows(n1, w, p + "mix.", m, eps)
            y = latent_attention(n1, w, p + "mix.", m, eps, kept[i if j is None else j])
        else:
            y = channel_delta(n1, w, p + "mix.", m, eps)
        ff = layer.get("mlp")
        if ff is not None:
            n2 = rms(x, w[p + "norm2"], eps)
            y = y + (dense_ff(n2, w, p + "mlp.") if ff["kind"] == "dense"
                     else table_moe(n2, tokens, w, p + "mlp.", ff["router"]["top"]))
        x = x + y
        stream.append(x)
    return rms(x, w["final.norm"], eps) @ w["head"].T, torch.stack(stream)
