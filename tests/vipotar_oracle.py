"""Plain implementation of the Vipotar design for tests: one function per mechanism, one sequence at a time, no cache, no
batching, no code shared with the package. ``cfg`` is the parsed config.json, ``w`` a dict of tensors by name. Everything
runs in the dtype of ``DT`` (float64 by default)."""

import math

import torch

DT = torch.float64


def rms(x, weight, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def frequencies(dims, base, scaling=None):
    """Angle per position of every rotated pair, and the factor on cosines and sines."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return f, 1.0
    s, orig = scaling["factor"], scaling["original"]

    def pair_of(turns):          # the (real-valued) pair index that makes ``turns`` rotations over the original length
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s * r + fi * (1.0 - r))
    return out, 0.1 * math.log(s) + 1.0


def rotate(x, rot, first_position=0):
    """x [T, heads, d]: values 2i and 2i + 1 of every head turn together, for the first ``dims`` values."""
    f, amp = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    out = x.clone()
    for p in range(x.shape[0]):
        for i, fi in enumerate(f):
            a = (first_position + p) * fi
            c, s = math.cos(a) * amp, math.sin(a) * amp
            u, v = x[p, :, 2 * i], x[p, :, 2 * i + 1]
            out[p, :, 2 * i] = u * c - v * s
            out[p, :, 2 * i + 1] = v * c + u * s
    return out


def softmax_with_zero_sink(s):
    """Rows of scores (-inf: not visible); the denominator has one extra term exp(0)."""
    top = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(-top))


def window_attention(q, k, v, scale, window):
    """q [T, H, d], k [T, G, d], v [T, G, dv], already rotated; a query sees itself and ``window - 1`` keys before it."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    i, j = torch.arange(T).view(T, 1), torch.arange(T).view(1, T)
    seen = (i >= j) if window is None else (i >= j) & (i - j < window)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = torch.where(seen, q[:, h] @ k[:, g].T * scale, torch.full((T, T), -math.inf, dtype=q.dtype))
        out[:, h] = softmax_with_zero_sink(s) @ v[:, g]
    return out


def left_mixer(h, w, p, m):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate((h @ w[p + "q"].T).view(T, H, d), m["rot"])
    k = rotate((h @ w[p + "k"].T).view(T, G, d), m["rot"])
    v = (h @ w[p + "v"].T).view(T, G, dv)
    o = window_attention(q, k, v, m["scale"], (m.get("mask") or {}).get("size"))
    return o.reshape(T, H * dv) @ w[p + "o"].T


def decayed_sum(q, k, v, decay, state=None):
    """q, k [T, H, d], v [T, H, dv], decay [H]: outputs [T, H, dv] and the state [H, d, dv] after the last token."""
    T, H = q.shape[:2]
    S = torch.zeros(H, q.shape[2], v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = decay.view(H, 1, 1) * S + k[t].unsqueeze(2) * v[t].unsqueeze(1)
        out.append((q[t].unsqueeze(2) * S).sum(1))
    return torch.stack(out), S


def right_mixer(h, w, p, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).view(T, H, d)
    k = silu(h @ w[p + "k"].T).view(T, H, d)
    v = silu(h @ w[p + "v"].T).view(T, H, dv)
    o, _ = decayed_sum(q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    return (rms(o.reshape(T, H * dv), w[p + "norm"], eps) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps):
    a, b = left_mixer(h, w, p + "left.", m["left"]), right_mixer(h, w, p + "right.", m["right"], eps)
    return (rms(a, w[p + "left.out"], eps) + rms(b, w[p + "right.out"], eps)) / 2.0


def dense_ff(h, w, p):
    return torch.clamp(h @ w[p + "up"].T, min=0.0) ** 2 @ w[p + "down"].T


def one_layer(x, w, p, layer, cfg):
    eps = cfg["norm"]["eps"]
    h = rms(x, w[p + "norm1"], eps)
    y = parallel_mixer(h, w, p + "mix.", layer["mixer"], eps)
    if layer.get("mlp") is not None:
        y = y + dense_ff(h, w, p + "mlp.")
    return x + cfg["residual_mult"] * y


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def forward(cfg, w, tokens):
    """Logits [T, vocab] and the residual stream after every layer run [runs, T, width]."""
    w = {k: v.to(DT) for k, v in w.items()}
    layers, loop = cfg["layers"], cfg.get("loop")
    first = w["embed"][[int(t) for t in tokens]]
    x, stream = first, []

    def run(i):
        nonlocal x
        x = one_layer(x, w, f"l{i}.", layers[i], cfg)
        stream.append(x)

    i = 0
    while i < len(layers):
        if loop is None or i != loop["start"]:
            run(i)
            i += 1
            continue
        for t in range(loop["times"]):
            x = x + w["loop.step"][t] if t == 0 else x + first + w["loop.step"][t]
            for j in range(loop["start"], loop["stop"]):
                run(j)
        i = loop["stop"]
    return softcap(rms(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T, cfg["logit_softcap"]), torch.stack(stream)
