"""Plain implementation of the Mavidra design for tests: one function per mechanism, one sequence at a time, no cache, no
batching, no code shared with the package. ``cfg`` is the parsed config.json, ``w`` a dict of tensors by name. Everything
runs in the dtype of ``DT`` (float64 by default)."""

import math

import torch

DT = torch.float64
ROUND = lambda x: x              # applied to the inputs and outputs of matrix products: tests set it to see what rounding does


def linear(x, w):
    return ROUND(ROUND(x) @ w.T)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def rms(x, weight, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def layer_norm(x, weight, bias, eps):
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * weight + bias


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def bigram_rows(tokens, spec):
    """Row of the bigram table for every token of a sequence."""
    rows, before = [], None
    for t in tokens:
        t = int(t)
        rows.append(spec["buckets"] if before is None else (before * spec["mul_prev"] + t * spec["mul_cur"]) % spec["buckets"])
        before = t
    return rows


def embedding(tokens, w, spec):
    x = w["embed"][[int(t) for t in tokens]] * spec["scale"]
    return x + w["bigram"][bigram_rows(tokens, spec["bigram"])]


def rotate(x, rot, first_position=0, halves=True):
    """x [T, heads, d]: pairs (i, i + dims / 2) of the first ``dims`` values turn (neighbours when not ``halves``)."""
    n = rot["dims"]
    i = torch.arange(n // 2)
    a = (first_position + torch.arange(x.shape[0], dtype=DT)).view(-1, 1) * float(rot["base"]) ** (-2.0 * i.to(DT) / max(n, 1))
    cos, sin = torch.cos(a).to(x.dtype).unsqueeze(1), torch.sin(a).to(x.dtype).unsqueeze(1)
    iu, iv = (i, i + n // 2) if halves else (2 * i, 2 * i + 1)
    u, v, out = x[..., iu], x[..., iv], x.clone()
    out[..., iu], out[..., iv] = u * cos - v * sin, v * cos + u * sin
    return out


def softmax(s, sink=None):
    """Rows of scores (-inf: not visible); a sink adds one exponential to the denominator only."""
    top = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    e = torch.exp(s - top)
    den = e.sum(dim=-1, keepdim=True)
    return e / (den if sink is None else den + torch.exp(sink - top))


def visible(T, window=None):
    i, j = torch.arange(T).view(T, 1), torch.arange(T).view(1, T)
    return (i >= j) if window is None else (i >= j) & (i - j < window)


def grouped_attention(q, k, v, scale, sink=None, window=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; sink [H]. Returns [T, H, dv]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    seen = visible(T, window)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = torch.where(seen, q[:, h] @ k[:, g].T * scale, torch.full((T, T), -math.inf, dtype=q.dtype))
        out[:, h] = softmax(s, None if sink is None else sink[h]) @ v[:, g]
    return out


def left_mixer(h, w, p, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate(rms(linear(h, w[p + "q"]).view(T, H, d), w[p + "q.norm"], eps), m["rot"])
    k = rotate(rms(linear(h, w[p + "k"]).view(T, G, d), w[p + "k.norm"], eps), m["rot"])
    v = linear(h, w[p + "v"]).view(T, G, dv)
    o = grouped_attention(q, k, v, m["scale"], w[p + "sink"])
    o = o * sigmoid(linear(h, w[p + "g"])).unsqueeze(2)
    return linear(o.reshape(T, H * dv), w[p + "o"])


def short_conv(x, taps):
    """x [T, C], taps [C, n]: the last tap meets the current token."""
    T, n = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(n):
            s = t - (n - 1) + j
            if s >= 0:
                out[t] += taps[:, j] * x[s]
    return out


def delta_scan(q, k, v, g, beta, state=None):
    """q, k [T, H, d], v [T, H, dv], g, beta [T, H]: outputs [T, H, dv] and the last state [H, d, dv]."""
    T, H = q.shape[:2]
    S = torch.zeros(H, q.shape[2], v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = S * g[t].view(H, 1, 1)
        u = beta[t].unsqueeze(1) * (v[t] - (S * k[t].unsqueeze(2)).sum(1))
        S = S + k[t].unsqueeze(2) * u.unsqueeze(1)
        out.append((S * q[t].unsqueeze(2)).sum(1))
    return torch.stack(out), S


def right_mixer(h, w, p, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv = lambda n: silu(short_conv(linear(h, w[p + n]), w[p + n + ".conv"]))
    group = torch.arange(H) // (H // G)
    q = unit(conv("q").view(T, G, d))[:, group] * d ** -0.5
    k = unit(conv("k").view(T, G, d))[:, group]
    v = conv("v").view(T, H, dv)
    beta = sigmoid(linear(h, w[p + "b"]))
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(linear(h, w[p + "a"]) + w[p + "dt_bias"]))
    o, _ = delta_scan(q, k, v, g, beta)
    o = rms(o, w[p + "norm"], eps) * silu(linear(h, w[p + "g"])).view(T, H, dv)
    return linear(o.reshape(T, H * dv), w[p + "o"])


def parallel_mixer(h, w, p, m, eps):
    return m["left_scale"] * left_mixer(h, w, p + "left.", m["left"], eps) + m["right_scale"] * right_mixer(h, w, p + "right.", m["right"], eps)


def gla_scan(q, k, v, alpha, state=None):
    """q, k, alpha [T, H, d], v [T, H, dv]: outputs [T, H, dv] and the last state [H, d, dv]."""
    T, H = q.shape[:2]
    S = torch.zeros(H, q.shape[2], v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = alpha[t].unsqueeze(2) * S + k[t].unsqueeze(2) * v[t].unsqueeze(1)
        out.append((S * q[t].unsqueeze(2)).sum(1))
    return torch.stack(out), S


def gla_mixer(h, w, p, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(h, w[p + "q"]).view(T, H, d) * d ** -0.5
    k = linear(h, w[p + "k"]).view(T, H, d)
    v = linear(h, w[p + "v"]).view(T, H, dv)
    z = linear(linear(h, w[p + "a1"]), w[p + "a2"]) + w[p + "a2.b"]
    alpha = torch.exp(-softplus(-z) / m["tau"]).view(T, H, d)            # sigmoid(z) ** (1 / tau)
    o, _ = gla_scan(q, k, v, alpha)
    o = rms(o, w[p + "norm"], eps).reshape(T, H * dv) * silu(linear(h, w[p + "g"]))
    return linear(o, w[p + "o"])


def latent_rows(h, w, p, m, eps):
    """What the cache keeps of a layer: the normed latent [T, kv_rank] and the rotated key part [T, rot_dim]."""
    kv = linear(h, w[p + "dkv"])
    c = rms(kv[:, : m["kv_rank"]], w[p + "dkv.norm"], eps)
    return c, rotate(kv[:, m["kv_rank"]:].unsqueeze(1), m["rot"], halves=False).squeeze(1)


def latent_mixer(h, w, p, m, eps, rows):
    """``rows``: the layer's own latent rows, or those of the layer it shares with."""
    T, H, d, r, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = rows
    q = linear(rms(linear(h, w[p + "dq"]), w[p + "dq.norm"], eps), w[p + "uq"]).view(T, H, d + r)
    q = torch.cat([q[..., :d], rotate(q[..., d:], m["rot"], halves=False)], 2)
    k = torch.cat([linear(c, w[p + "uk"]).view(T, H, d), kr.unsqueeze(1).expand(T, H, r)], 2)
    v = linear(c, w[p + "uv"]).view(T, H, dv)
    o = grouped_attention(q, k, v, m["scale"], window=m["mask"]["size"])
    o = o * sigmoid(linear(h, w[p + "g"])).unsqueeze(2)
    return linear(o.reshape(T, H * dv), w[p + "o"])


def choose(scores, correction, router):
    """scores [E] of one token -> the chosen experts, best choice score first."""
    choice = scores + correction
    E, n = choice.shape[0], router["groups"]["count"]
    size = E // n
    groups = []
    for g in range(n):
        best = sorted((float(c) for c in choice[g * size: (g + 1) * size]), reverse=True)
        groups.append((-sum(best[:2]), g))
    kept = {g for _, g in sorted(groups)[: router["groups"]["keep"]]}
    open_ = [e for e in range(E) if e // size in kept]
    return sorted(open_, key=lambda e: (-float(choice[e]), e))[: router["top"]]


def choice_margin(scores, correction, router):
    """How far the nearest other choice of experts is, in choice scores: what an implementation that rounds may get wrong."""
    choice, n = scores + correction, router["groups"]["count"]
    size, keep, top = choice.shape[0] // n, router["groups"]["keep"], router["top"]
    best = torch.stack([choice[g * size: (g + 1) * size].sort(descending=True).values[:2].sum() for g in range(n)])
    order = best.argsort(descending=True)
    gap = best[order[keep - 1]] - best[order[keep]] if keep < n else torch.tensor(math.inf)
    open_ = torch.cat([choice[g * size: (g + 1) * size] for g in order[:keep]]).sort(descending=True).values
    return min(float(gap), float(open_[top - 1] - open_[top]) if top < len(open_) else math.inf)


def moe(h, w, p, ff):
    h = ROUND(h)
    s = sigmoid(h @ w[p + "router"].T)
    rows = []
    for t in range(h.shape[0]):
        y = torch.zeros(h.shape[1], dtype=h.dtype)
        for e in choose(s[t], w[p + "correction"], ff["router"]):
            a = silu(linear(h[t], w[f"{p}e{e}.gate"])) * linear(h[t], w[f"{p}e{e}.up"])
            y = y + s[t, e] * linear(a, w[f"{p}e{e}.down"])
        rows.append(y)
    return torch.stack(rows)


def forward(cfg, w, tokens):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    w = {k: (v if v.dtype == torch.int32 else v.to(DT)) for k, v in w.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    norm = lambda x, n: layer_norm(x, w[n], w[n + ".b"], eps)
    x, stream, latents = embedding(tokens, w, cfg["embedding"]), [], {}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        h = norm(x, p + "norm1")
        if l["type"] == "parallel":
            y = parallel_mixer(h, w, p + "mix.", m, eps)
        elif l["type"] == "gla":
            y = gla_mixer(h, w, p + "mix.", m, eps)
        else:
            j = m.get("kv_from")
            if j is None:
                latents[i] = latent_rows(h, w, p + "mix.", m, eps)
            y = latent_mixer(h, w, p + "mix.", m, eps, latents[i if j is None else j])
        x = x + mult * norm(y, p + "norm1b")
        if l.get("mlp") is not None:
            x = x + mult * norm(moe(norm(x, p + "norm2"), w, p + "mlp.", l["mlp"]), p + "norm2b")
        stream.append(x)
    return linear(norm(x, "final.norm"), w["embed"]), torch.stack(stream)
