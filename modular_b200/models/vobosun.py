"""Vobosun: a decoder of softmax-attention and generalized delta-rule layers whose norms are elementwise (dynamic tanh).

Every layer is ``x += T(mixer(shift(T(x))))`` and then ``x += T(ff(T(x)))`` on an fp32 residual stream, with
``T(y) = tanh(alpha * y) * w + b`` (weights of its own each time). The mixer's input moves towards that of the token before by a
factor per channel. The mixer is grouped softmax attention with biases and partial rotation
(:mod:`modular_b200.nn.window_attention`) or a generalized delta rule (:mod:`modular_b200.nn.general_delta`); the feed-forward is
dense with the xIELU activation, or a mixture of experts with a softmax router, identity experts and a shared expert
(:class:`modular_b200.nn.moe.ScoreRouter`). ``config.json`` lists the layers one by one, each with its own sizes; a layer may use the
weights of another one, with a cache and a state of its own.

Cache: one key/value plane per attention layer in the paged cache; recurrent states and every layer's last normed row in state
slots. The seam between two branches is one kernel (:func:`modular_b200.nn.residual.tanh_seam`). Decode steps replay CUDA graphs.
"""

from __future__ import annotations

import json
import math
from dataclasses import dataclass, field
from typing import Optional

import torch

from .. import ops
from ..nn.delta_rule import gemm_k, pad_to, up8
from ..nn.general_delta import GeneralDelta, GeneralDeltaConfig
from ..nn.moe import ScoreRouter, ScoreRouterConfig, expert_mlp, gated_mlp
from ..nn.residual import tanh_seam
from ..nn.rotary_embedding import RopeScaling, cos_sin_table
from ..nn.window_attention import WindowAttention, WindowAttentionConfig, head_width, tensor_core_plan
from .decode_graphs import DecodeGraphs

ATTENTION, DELTA = "attention", "general_delta"


@dataclass
class VobosunConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: tuple                                   # the entries of config.json's ``layers``
    max_position_embeddings: int = 1 << 17
    architectures: tuple = ("Vobosun",)
    raw: dict = field(default_factory=dict, repr=False)

    def __post_init__(self):
        if not self.layers:
            raise ValueError("config.json lists no layers")
        for i, l in enumerate(self.layers):
            j, ff = l.get("weights_of"), l.get("mlp")
            if l["type"] not in (ATTENTION, DELTA):
                raise ValueError(f"layer {i}: mixer type {l['type']!r} is not known")
            if ff is not None and ff["kind"] not in ("dense", "moe"):
                raise ValueError(f"layer {i}: feed-forward kind {ff['kind']!r} is not known")
            try:
                if l["type"] == ATTENTION:
                    self.attention(i)
                if ff is not None and ff["kind"] == "moe":
                    self.router(i)
            except ValueError as e:
                raise ValueError(f"layer {i}: {e}") from None
            if j is not None:
                rest = lambda e: {k: v for k, v in e.items() if k != "weights_of"}
                if not 0 <= j < len(self.layers) or j == i or self.layers[j].get("weights_of") is not None or rest(l) != rest(self.layers[j]):
                    raise ValueError(f"layer {i}: weights_of must name a layer with weights of its own and the same sizes")

    # what the generic engine code asks of any config
    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def num_attention_heads(self) -> int:
        return max(l["mixer"]["heads"] for l in self.layers)

    @property
    def num_key_value_heads(self) -> int:
        return self.num_attention_heads        # the batch packer's tile plan is not used here

    @property
    def width_pad(self) -> int:
        return gemm_k(self.hidden_size)

    @classmethod
    def from_hf(cls, d: dict) -> "VobosunConfig":
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), norm_eps=float(d["norm"]["eps"]), layers=tuple(d["layers"]),
                   max_position_embeddings=int(d.get("max_position_embeddings", 1 << 17)), raw=dict(d))

    def to_hf(self) -> dict:
        return {"architecture": "Vobosun", "architectures": list(self.architectures), "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.norm_eps}, "layers": json.loads(json.dumps(list(self.layers)))}

    # ------------------------------------------------------------ layers
    def of_type(self, kind: str) -> tuple:
        return tuple(i for i, l in enumerate(self.layers) if l["type"] == kind)

    def source(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses."""
        j = self.layers[i].get("weights_of")
        return i if j is None else j

    def attention(self, i: int) -> WindowAttentionConfig:
        m = self.layers[i]["mixer"]
        rot = m.get("rot") or {}
        factor = float((rot.get("scaling") or {}).get("factor", 1.0))
        return WindowAttentionConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), int(rot.get("dims", 0)),
                                     float(rot.get("base", 1e4)), RopeScaling("linear", factor), halves=True, bias=True)

    def delta(self, i: int, rank: int = 0) -> GeneralDeltaConfig:
        m = self.layers[i]["mixer"]
        return GeneralDeltaConfig(m["heads"], m["dim"], rank, self.norm_eps)

    def is_moe(self, i: int) -> bool:
        ff = self.layers[i].get("mlp")
        return ff is not None and ff["kind"] == "moe"

    def router(self, i: int) -> ScoreRouterConfig:
        r = self.layers[i]["mlp"]["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        return ScoreRouterConfig(int(r["experts"]), int(r["top"]), int(g["count"]), int(g["keep"]), renormalize=True, softmax=True,
                                 group_max=True, identity=int(r.get("identity") or 0))

    # ------------------------------------------------------------ cache
    @property
    def head_width(self) -> int:
        return head_width(max([max(self.attention(i).dim, self.attention(i).vdim) for i in self.of_type(ATTENTION)], default=8))

    @property
    def cache_heads(self) -> int:
        return max([self.attention(i).kv_heads for i in self.of_type(ATTENTION)], default=1)

    def state_specs(self) -> tuple:
        out = []
        for i, l in enumerate(self.layers):
            out.append((f"l{i}.shift", (self.width_pad,), torch.float32))
            if l["type"] == DELTA:
                out += [(f"l{i}.{name}", shape, torch.float32) for name, shape in self.delta(i).state_shapes().items()]
        return tuple(out)

    # ------------------------------------------------------------ checkpoint
    def tensor_shapes(self, ranks: Optional[dict] = None) -> dict:
        """Name -> shape of every tensor of a checkpoint. ``ranks``: rank of the decay projection per delta-rule layer (not in the
        config; a checkpoint's shapes give it, 16 otherwise)."""
        W, out = self.hidden_size, {"embed": (self.vocab_size, self.hidden_size)}

        def norm(name):
            out.update({name: (W,), name + ".b": (W,), name + ".alpha": ()})

        for i, l in enumerate(self.layers):
            if self.source(i) != i:
                continue
            m, p, q, ff = l["mixer"], f"l{i}.mix.", f"l{i}.mlp.", l.get("mlp")
            norm(f"l{i}.norm1")
            norm(f"l{i}.norm1b")
            out[f"l{i}.shift"] = (W,)
            if l["type"] == ATTENTION:
                for n, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                    out.update({p + n: (rows, W), p + n + ".b": (rows,)})
                out[p + "o"] = (W, m["heads"] * m["vdim"])
            else:
                n, r = m["heads"] * m["dim"], (ranks or {}).get(i, 16)
                out.update({p + k: (n, W) for k in "rkvga"})
                out.update({p + "a.b": (n,), p + "w1": (r, W), p + "w2": (n, r), p + "w0": (n,), p + "norm": (n,), p + "o": (W, n)})
            if ff is None:
                continue
            norm(f"l{i}.norm2")
            norm(f"l{i}.norm2b")
            if ff["kind"] == "dense":
                out.update({q + "up": (ff["ff"], W), q + "down": (W, ff["ff"]), q + "act": (2,)})
                continue
            c = self.router(i)
            gated = [(f"{q}e{e}.", ff["expert"]["ff"]) for e in range(c.experts)]
            gated += [(q + "shared.", ff["shared"]["ff"])] if ff.get("shared") else []
            for n, F in gated:
                out.update({n + "gate": (F, W), n + "up": (F, W), n + "down": (W, F)})
            out.update({q + "router": (c.candidates, W), q + "correction": (c.candidates,)})
        norm("final.norm")
        out["head"] = (self.vocab_size, W)
        return out

    def param_count(self) -> int:
        return sum(math.prod(shape) for shape in self.tensor_shapes().values())

    @classmethod
    def build(cls, width: int, vocab: int, pattern: str, attention: dict, delta: dict, ff: int, expert_ff: int = 0, router: Optional[dict] = None,
              shared_ff: int = 0, eps: float = 1e-6) -> "VobosunConfig":
        """A config from a pattern of layers: ``A`` attention, ``D`` delta rule with a dense feed-forward, ``M`` attention, ``E`` delta
        rule with experts; a digit repeats the layer of that index with its weights, a lower-case letter has no feed-forward."""
        layers, copy = [], lambda d: json.loads(json.dumps(d))
        for ch in pattern:
            if ch.isdigit():
                layers.append({**copy(layers[int(ch)]), "weights_of": int(ch)})
                continue
            kind = ch.upper()
            mlp = {"kind": "dense", "ff": ff}
            if kind in "ME":
                mlp = {"kind": "moe", "expert": {"ff": expert_ff}, "router": copy(router)}
                if shared_ff:
                    mlp["shared"] = {"ff": shared_ff}
            layers.append({"type": ATTENTION if kind in "AM" else DELTA, "mixer": copy(attention if kind in "AM" else delta),
                           "mlp": mlp if ch.isupper() else None})
        return cls(vocab, width, eps, tuple(layers))

    @classmethod
    def tiny(cls, **kw) -> "VobosunConfig":
        base = dict(width=160, vocab=512, pattern="AEMD1a", ff=240, expert_ff=80, shared_ff=112,
                    router=dict(experts=7, top=3, identity=2, groups=dict(count=3, keep=2)),
                    attention=dict(heads=6, kv_heads=2, dim=40, vdim=24, scale=40 ** -0.5,
                                   rot=dict(base=20000.0, dims=32, scaling=dict(factor=2.0))),
                    delta=dict(heads=3, dim=40))
        base.update(kw)
        return cls.build(**base)


@dataclass
class VobosunLayer:
    norm1: tuple                                   # (alpha, weight, bias) of the elementwise norms
    norm1b: tuple
    shift: torch.Tensor
    mixer: object                                  # WindowAttention | GeneralDelta
    norm2: Optional[tuple] = None
    norm2b: Optional[tuple] = None
    xielu: Optional[tuple] = None                  # dense: factors of the activation
    w_up: Optional[torch.Tensor] = None            # dense: [ff, width]; experts: gate and up [E, 2 ff, width]
    w_down: Optional[torch.Tensor] = None          # dense: [width, ff]; experts: [E, width, ff]
    router: Optional[ScoreRouter] = None
    shared_up: Optional[torch.Tensor] = None       # shared expert: gate and up [2 ff, width]
    shared_down: Optional[torch.Tensor] = None


def xielu_factors(act) -> tuple:
    """Stored (p, q) -> the factors of z^2 above zero and of exp(z) - 1 - z below."""
    softplus = lambda z: max(z, 0.0) + math.log1p(math.exp(-abs(z)))
    p, q = (float(v) for v in act)
    return softplus(p), 0.5 + softplus(q)


class VobosunWeights:
    def __init__(self, cfg: VobosunConfig, embed, layers, final_norm, head):
        self.cfg, self.embed, self.layers, self.final_norm, self.head = cfg, embed, layers, final_norm, head

    @classmethod
    def from_state_dict(cls, cfg: VobosunConfig, sd: dict, device="cpu", dtype=torch.bfloat16) -> "VobosunWeights":
        W, Wp = cfg.hidden_size, cfg.width_pad
        ranks = {i: sd[f"l{i}.mix.w1"].shape[0] for i in cfg.of_type(DELTA) if f"l{i}.mix.w1" in sd}
        for name, shape in cfg.tensor_shapes(ranks).items():
            if name not in sd:
                raise KeyError(f"the checkpoint has no tensor {name!r}")
            if tuple(sd[name].shape) != tuple(shape):
                raise ValueError(f"{name}: {tuple(sd[name].shape)} in the checkpoint, {tuple(shape)} by the config")
        put = lambda t: t.to(device=device, dtype=dtype).contiguous()
        vector = lambda n: put(torch.nn.functional.pad(sd[n], (0, Wp - W)))
        norm = lambda n: (float(sd[n + ".alpha"]), vector(n), vector(n + ".b"))
        layers: list = [None] * len(cfg.layers)

        def gated(prefix, F):
            return torch.cat([pad_to(sd[prefix + n], F, Wp) for n in ("gate", "up")]), pad_to(sd[prefix + "down"], Wp, F)

        for i, l in enumerate(cfg.layers):
            if cfg.source(i) != i:
                continue
            p, q, ff = f"l{i}.mix.", f"l{i}.mlp.", l.get("mlp")
            t = {k[len(p):]: v for k, v in sd.items() if k.startswith(p)}
            mixer = (WindowAttention(cfg.attention(i), t, cfg.head_width, Wp, device, dtype) if l["type"] == ATTENTION else
                     GeneralDelta(cfg.delta(i, ranks[i]), t, Wp, device, dtype))
            if l["type"] == ATTENTION:
                mixer.w_in = put(mixer.w_in)
            lw = layers[i] = VobosunLayer(norm(f"l{i}.norm1"), norm(f"l{i}.norm1b"), vector(f"l{i}.shift"), mixer)
            if ff is None:
                continue
            lw.norm2, lw.norm2b = norm(f"l{i}.norm2"), norm(f"l{i}.norm2b")
            if ff["kind"] == "dense":
                F = gemm_k(ff["ff"])
                lw.w_up, lw.w_down, lw.xielu = put(pad_to(sd[q + "up"], F, Wp)), put(pad_to(sd[q + "down"], Wp, F)), xielu_factors(sd[q + "act"])
                continue
            c, F = cfg.router(i), gemm_k(ff["expert"]["ff"])
            lw.router = ScoreRouter(c, sd[q + "router"], sd[q + "correction"], Wp, device, dtype)
            experts = [gated(f"{q}e{e}.", F) for e in range(c.experts)]
            lw.w_up, lw.w_down = (put(torch.stack([e[k] for e in experts])) for k in (0, 1))
            if ff.get("shared"):
                lw.shared_up, lw.shared_down = (put(w) for w in gated(q + "shared.", gemm_k(ff["shared"]["ff"])))
        layers = [layers[cfg.source(i)] for i in range(len(layers))]
        return cls(cfg, put(pad_to(sd["embed"], up8(cfg.vocab_size), Wp)), layers, norm("final.norm"),
                   put(pad_to(sd["head"], up8(cfg.vocab_size), Wp)))

    @staticmethod
    def random_state_dict(cfg: VobosunConfig, seed: int = 0, dtype=torch.float32, device="cpu") -> dict:
        """Random tensors of a checkpoint: projections scaled by their fan-in, norms around one."""
        g = torch.Generator(device=device).manual_seed(seed)
        sd = {}
        for name, shape in cfg.tensor_shapes().items():
            leaf, t = name.rsplit(".", 1)[-1], torch.randn(shape, generator=g, device=device)
            if leaf == "alpha":
                t = 0.7 + 0.1 * t
            elif leaf in ("b", "correction"):
                t = 0.1 * t
            elif leaf == "shift":
                t = torch.sigmoid(t)
            elif "norm" in leaf:
                t = 1.0 + 0.1 * t
            elif name != "embed" and leaf not in ("w0", "act"):
                t = t * shape[-1] ** -0.5
            sd[name] = t.to(dtype)
        return sd

    @classmethod
    def random_init(cls, cfg: VobosunConfig, device="cpu", dtype=torch.bfloat16, seed: int = 0) -> "VobosunWeights":
        """Random weights, generated on ``device``."""
        return cls.from_state_dict(cfg, cls.random_state_dict(cfg, seed, dtype, device), device, dtype)


class VobosunModel:
    """Serves :class:`VobosunConfig` behind the engine's model interface (``forward_tensors``); decode steps replay CUDA graphs.
    ``kv_cache``: [pages, 2, attention layers, kv heads, page, head width]; ``state``: the cache manager's state tensors."""

    use_executor = False
    executor = None
    logits_buf = None

    def __init__(self, cfg: VobosunConfig, weights: VobosunWeights, kv_cache: torch.Tensor, max_tokens: int = 8192,
                 max_seqs: int = 256, max_position: Optional[int] = None, state: Optional[dict] = None):
        self.cfg, self.w, self.kv, self.state = cfg, weights, kv_cache, state or {}
        self.device, self.dtype = weights.embed.device, weights.embed.dtype
        self.max_tokens, self.max_seqs = max_tokens, max_seqs
        self.page_size = kv_cache.shape[4]
        self.max_position = max_position or min(cfg.max_position_embeddings, 1 << 17)
        self.plane = {i: j for j, i in enumerate(cfg.of_type(ATTENTION))}
        tables: dict = {}
        self.cos_sin = {}
        for i in self.plane:
            a = cfg.attention(i)
            key = (a.rot_dims, a.rope_base, a.rope_scaling.factor)
            if key not in tables:
                tables[key] = cos_sin_table(a.rot_dims, self.max_position, a.rope_base, a.rope_scaling, self.device) if a.rot_dims else None
            self.cos_sin[i] = tables[key]
        self.groups = sorted({cfg.attention(i).group_pad for i in self.plane})
        self.moe_layers = [i for i in range(len(cfg.layers)) if cfg.is_moe(i)]
        self.max_experts = max([cfg.router(i).experts for i in self.moe_layers], default=0)
        self.graphs: Optional[DecodeGraphs] = None
        self.forward_calls = 0

    # ------------------------------------------------------------ CUDA graphs of decode steps
    def capture_decode_graphs(self, batch_sizes) -> None:
        if self.device.type != "cuda":
            return
        if self.graphs is None:
            self.graphs = DecodeGraphs(self._forward, self.device,
                                       -(-min(self.max_position, self.kv.shape[0] * self.page_size) // self.page_size), self.max_seqs)
        self.graphs.capture(batch_sizes)

    @property
    def graph_replays(self) -> int:
        return self.graphs.replays if self.graphs is not None else 0

    @property
    def replayed_calls(self) -> int:
        return self.graphs.replayed_calls if self.graphs is not None else 0

    @torch.no_grad()
    def forward_tensors(self, tokens, positions, slots, block_table, q_start, q_len, kv_len, logit_rows, plan=None,
                        state_slot=None, lora=None) -> torch.Tensor:
        """fp32 logits [len(logit_rows), vocab] of a ragged step."""
        if lora is not None:
            raise ValueError("LoRA adapters are not implemented for this family")
        self.forward_calls += 1
        if self.graphs is not None:
            size = self.graphs.fits(tokens.shape[0], q_len.shape[0], logit_rows.shape[0])
            if size:
                return self.graphs.replay(size, block_table, tokens=tokens, positions=positions, slots=slots, kv_len=kv_len,
                                          state_slot=state_slot)
        return self._forward(tokens, positions, slots, block_table, q_start, q_len, kv_len, logit_rows, state_slot)

    # ------------------------------------------------------------ step
    @torch.no_grad()
    def _forward(self, tokens, positions, slots, block_table, q_start, q_len, kv_len, logit_rows, state_slot=None,
                 stream: Optional[list] = None) -> torch.Tensor:
        """``stream`` (a list) collects a copy of the residual stream after every layer."""
        c, w, T, Wp, dev, lin = self.cfg, self.w, tokens.shape[0], self.cfg.width_pad, self.device, ops.linear
        new = lambda rows: torch.empty(rows, Wp, dtype=self.dtype, device=dev)
        one_token = T == q_len.shape[0]
        plans = {g: tensor_core_plan(g, self.kv.shape[5], self.dtype, self.page_size, q_start, q_len, T, one_token)
                 for g in self.groups}
        counts = torch.zeros(len(self.moe_layers), self.max_experts, dtype=torch.int32, device=dev)
        # the shifted seam of a mixer reads one buffer of the stream and writes the other
        x, other = torch.empty(2, T, Wp, dtype=torch.float32, device=dev)
        # what the next seam adds to the stream: the embedding first, then one branch at a time
        pending = dict(ids=tokens, table=w.embed)
        routed = 0
        for i, l in enumerate(w.layers):
            h = new(T)
            tanh_seam(x=x if i else None, x_out=other, norm1=l.norm1, n1=h, shift=l.shift, prev=self.state[f"l{i}.shift"],
                      state_idx=state_slot, q_start=q_start, q_len=q_len, kv_len=kv_len, **pending)
            x, other = other, x
            if c.layers[i]["type"] == DELTA:
                y = l.mixer(h, lin, self.state[f"l{i}.gdelta"], state_slot, q_start, q_len, kv_len, one_token)
            else:
                px = lin(h, l.mixer.w_in)
                l.mixer.prep(px, positions, self.cos_sin[i], slots, self.kv, self.plane[i])
                o = l.mixer(px[:, : l.mixer.k_off], self.kv, self.plane[i], block_table, q_start, q_len, kv_len, plans[l.mixer.cfg.group_pad])
                y = lin(o, l.mixer.w_o)
            pending = dict(a=y, norm_u=l.norm1b)
            if l.norm2 is not None:
                h = new(T)
                tanh_seam(x=x, x_out=x, norm1=l.norm2, n1=h, **pending)
                pending = dict(norm_u=l.norm2b)
                if l.router is None:
                    pending["a"] = lin(ops.xielu(lin(h, l.w_up), *l.xielu), l.w_down)
                else:
                    rows, offsets, inverse, pair_w = l.router.route(h, counts[routed, : l.router.cfg.experts])
                    routed += 1
                    pending.update(e=expert_mlp(rows, offsets, l.w_up, l.w_down, T), inverse=inverse, pair_w=pair_w,
                                   self_rows=h if l.router.cfg.identity else None)
                    if l.shared_up is not None:
                        pending["a"] = gated_mlp(h, l.shared_up, l.shared_down)
            if stream is not None:
                tanh_seam(x=x, x_out=x, **pending)
                stream.append(x[:, : c.hidden_size].clone())
                pending = {}
        out = new(logit_rows.shape[0])
        if out.shape[0] == 0:
            return torch.empty(0, c.vocab_size, dtype=torch.float32, device=dev)
        tanh_seam(x=x, rows=logit_rows, norm1=w.final_norm, n1=out, **pending)
        logits = lin(out, w.head, out_dtype=torch.float32)
        return logits if logits.shape[1] == c.vocab_size else logits[:, : c.vocab_size].contiguous()
