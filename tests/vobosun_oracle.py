"""Plain implementation of the Vobosun design for tests: one function per mechanism, one sequence at a time, no cache, no
batching, no code shared with the package. ``cfg`` is the parsed config.json, ``w`` a dict of tensors by name. Everything
runs in the dtype of ``DT`` (float64 by default)."""

import math

import torch

DT = torch.float64
ROUND = lambda x: x              # applied to the inputs and outputs of matrix products: tests set it to see what rounding does


def linear(x, w, bias=None):
    y = ROUND(x) @ w.T
    return ROUND(y if bias is None else y + bias)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def dynamic_tanh(x, alpha, weight, bias):
    return torch.tanh(alpha * x) * weight + bias


def token_shift(h, mix, before=None):
    """Every row moves by ``mix`` towards the row before it; ``before``: the row ahead of the first one (None: zeros)."""
    out = torch.empty_like(h)
    prev = torch.zeros_like(h[0]) if before is None else before
    for t in range(h.shape[0]):
        out[t] = h[t] + (prev - h[t]) * mix
        prev = h[t]
    return out


def frequencies(rot):
    """Angle per position of every pair."""
    n = rot["dims"]
    f = float(rot["base"]) ** (-2.0 * torch.arange(n // 2, dtype=torch.float64) / max(n, 1))
    return (f / float((rot.get("scaling") or {}).get("factor", 1.0))).to(DT)


def rotate(x, rot, first_position=0):
    """x [T, heads, d]: pairs (i, i + dims / 2) of the first ``dims`` values turn."""
    n = rot["dims"]
    a = (first_position + torch.arange(x.shape[0], dtype=DT)).view(-1, 1, 1) * frequencies(rot)
    c, s, out = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype), x.clone()
    u, v = x[..., : n // 2], x[..., n // 2: n]
    out[..., : n // 2], out[..., n // 2: n] = u * c - v * s, v * c + u * s
    return out


def softmax(s):
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


def attention(q, k, v, scale):
    """q [T, H, d], k [T, G, d], v [T, G, dv], every row sees those at or before it: [T, H, dv]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for t in range(T):
            out[t, h] = softmax((k[: t + 1, g] @ q[t, h]) * scale) @ v[: t + 1, g]
    return out


def attention_mixer(h, w, p, m):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    project = lambda n, heads, width: linear(h, w[p + n], w[p + n + ".b"]).view(T, heads, width)
    q, k, v = project("q", H, d), project("k", G, d), project("v", G, dv)
    if m.get("rot"):
        q, k = rotate(q, m["rot"]), rotate(k, m["rot"])
    return linear(attention(q, k, v, m["scale"]).reshape(T, H * dv), w[p + "o"])


def general_delta_scan(r, k, v, decay, rate, state=None):
    """r, k, decay, rate [T, H, d], v [T, H, dv]: outputs [T, H, dv] and the last state [H, d, dv]."""
    T, H, d = k.shape
    S = torch.zeros(H, d, v.shape[2], dtype=k.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        new, o = torch.empty_like(S), []
        for h in range(H):
            u = k[t, h] / torch.sqrt((k[t, h] ** 2).sum() + 1e-6)
            change = torch.diag(decay[t, h]) - torch.outer(rate[t, h] * u, u)
            new[h] = change @ S[h] + torch.outer(k[t, h], v[t, h])
            o.append(new[h].T @ r[t, h])
        S = new
        out.append(torch.stack(o))
    return torch.stack(out), S


def general_delta_mixer(h, w, p, m, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    heads = lambda x: x.view(T, H, d)
    r, k, v = (heads(linear(h, w[p + n])) for n in "rkv")
    z = linear(torch.tanh(linear(h, w[p + "w1"])), w[p + "w2"]) + w[p + "w0"]
    decay = torch.exp(-math.exp(-0.5) * sigmoid(z))
    rate = sigmoid(linear(h, w[p + "a"]) + w[p + "a.b"])
    o, _ = general_delta_scan(r, k, v, heads(decay), heads(rate))
    o = o / torch.sqrt((o * o).mean(dim=-1, keepdim=True) + eps)
    return linear(o.reshape(T, H * d) * w[p + "norm"] * sigmoid(linear(h, w[p + "g"])), w[p + "o"])


def xielu(z, p, q):
    up = softplus(p) * z * z + 0.5 * z
    n = torch.clamp(z, max=0.0)
    down = (0.5 + softplus(q)) * (torch.expm1(n) - n) + 0.5 * z
    return torch.where(z > 0, up, down)


def dense(h, w, p):
    return linear(xielu(linear(h, w[p + "up"]), w[p + "act"][0], w[p + "act"][1]), w[p + "down"])


def gated(h, w, p):
    return linear(silu(linear(h, w[p + "gate"])) * linear(h, w[p + "up"]), w[p + "down"])


def choose(scores, correction, router):
    """scores [E] of one token -> the chosen experts, best choice score first."""
    choice, E = scores + correction, scores.shape[0]
    open_ = list(range(E))
    if router.get("groups"):
        n, keep = router["groups"]["count"], router["groups"]["keep"]
        size = E // n
        order = sorted(range(n), key=lambda g: (-float(choice[g * size: (g + 1) * size].max()), g))
        open_ = [e for e in open_ if e // size in order[:keep]]
    return sorted(open_, key=lambda e: (-float(choice[e]), e))[: router["top"]]


def choice_margin(scores, correction, router):
    """How far the nearest other choice of experts is, in choice scores: what an implementation that rounds may get wrong."""
    choice, top, gap = scores + correction, router["top"], math.inf
    g = router.get("groups")
    if g and g["keep"] < g["count"]:
        best = choice.view(g["count"], -1).max(1).values
        order = best.argsort(descending=True)
        gap = float(best[order[g["keep"] - 1]] - best[order[g["keep"]]])
        choice = choice.view(g["count"], -1)[order[: g["keep"]]].flatten()
    open_ = choice.sort(descending=True).values
    return min(gap, float(open_[top - 1] - open_[top]) if top < len(open_) else math.inf)


def router_scores(h, w, p):
    z = ROUND(h) @ w[p + "router"].T
    return softmax(z)


def moe(h, w, p, ff):
    s, real, rows = router_scores(h, w, p), ff["router"]["experts"], []
    for t in range(h.shape[0]):
        chosen = choose(s[t], w[p + "correction"], ff["router"])
        total = sum(s[t, e] for e in chosen) + 1e-20
        y = torch.zeros_like(h[t])
        for e in chosen:
            y = y + s[t, e] / total * (gated(h[t], w, f"{p}e{e}.") if e < real else ROUND(h[t]))
        rows.append(y)
    y = torch.stack(rows)
    return y + gated(h, w, p + "shared.") if ff.get("shared") else y


def forward(cfg, w, tokens):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    w = {k: (v if v.dtype == torch.int32 else v.to(DT)) for k, v in w.items()}
    eps, stream = cfg["norm"]["eps"], []
    norm = lambda x, n: dynamic_tanh(x, w[n + ".alpha"], w[n], w[n + ".b"])
    x = w["embed"][[int(t) for t in tokens]]
    for i, l in enumerate(cfg["layers"]):
        p, m, ff = f"l{l.get('weights_of', i)}.", l["mixer"], l.get("mlp")
        h = token_shift(norm(x, p + "norm1"), w[p + "shift"])
        y = attention_mixer(h, w, p + "mix.", m) if l["type"] == "attention" else general_delta_mixer(h, w, p + "mix.", m, eps)
        x = x + norm(y, p + "norm1b")
        if ff is not None:
            h = norm(x, p + "norm2")
            x = x + norm(dense(h, w, p + "mlp.") if ff["kind"] == "dense" else moe(h, w, p + "mlp.", ff), p + "norm2b")
        stream.append(x)
    return linear(norm(x, "final.norm"), w["head"]), torch.stack(stream)
