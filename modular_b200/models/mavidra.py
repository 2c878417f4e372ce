"""Mavidra: a decoder that mixes three kinds of layers, each followed by a routed mixture of experts, with norms on both sides of
every branch.

Every layer is ``x += m norm(mixer(norm(x)))`` and then ``x += m norm(experts(norm(x)))``, layer norms on an fp32 residual stream.
The mixer is gated linear attention (:mod:`modular_b200.nn.gated_linear_attention`), latent attention with a sliding window
(:mod:`modular_b200.nn.latent_attention`; a layer may read the cache rows of an earlier one), or softmax attention beside a gated
delta rule (:mod:`modular_b200.nn.parallel_mixer`). Experts are chosen by sigmoid scores within the best groups
(:class:`modular_b200.nn.moe.ScoreRouter`). The embedding adds rows of a bigram table and is also the output matrix.
``config.json`` lists the layers one by one, each with its own sizes.

Cache: keys and values of the softmax layers in the paged cache, one plane each; latent rows in a second paged tensor of the same
pages; recurrent states, convolution tails and the last token in state slots. The seam between two branches is one kernel
(:func:`modular_b200.nn.residual.sandwich_norm`). Decode steps replay CUDA graphs.
"""

from __future__ import annotations

import json
from dataclasses import dataclass, field
from typing import Optional

import torch

from .. import ops
from ..nn.bigram import STATE as BIGRAM_STATE
from ..nn.bigram import BigramConfig, bigram_rows
from ..nn.delta_rule import DeltaRule, DeltaRuleConfig, gemm_k, pad_to, up8
from ..nn.gated_linear_attention import GatedLinearAttention, GatedLinearConfig
from ..nn.latent_attention import LatentAttention, LatentAttentionConfig
from ..nn.moe import ScoreRouter, ScoreRouterConfig, expert_mlp
from ..nn.parallel_mixer import ParallelMixer
from ..nn.residual import sandwich_norm
from ..nn.rotary_embedding import cos_sin_table
from ..nn.window_attention import WindowAttention, WindowAttentionConfig, head_width, tensor_core_plan
from .decode_graphs import DecodeGraphs

GLA, LATENT, PARALLEL = "gla", "latent_attention", "parallel"


@dataclass
class MavidraConfig:
    vocab_size: int
    hidden_size: int
    embedding_scale: float
    norm_eps: float
    layers: tuple                                   # the entries of config.json's ``layers``
    bigram: Optional[BigramConfig] = None
    residual_mult: float = 1.0
    max_position_embeddings: int = 1 << 17
    architectures: tuple = ("Mavidra",)
    raw: dict = field(default_factory=dict, repr=False)

    def __post_init__(self):
        if not self.layers:
            raise ValueError("config.json lists no layers")
        for i, l in enumerate(self.layers):
            m, ff = l["mixer"], l.get("mlp")
            if l["type"] not in (GLA, LATENT, PARALLEL):
                raise ValueError(f"layer {i}: mixer type {l['type']!r} is not known")
            if ff is not None and ff["kind"] != "moe":
                raise ValueError(f"layer {i}: feed-forward kind {ff['kind']!r} is not known")
            try:
                if l["type"] == PARALLEL:
                    self.attention(i)
                    if m["right"]["heads"] % m["right"]["kv_heads"]:
                        raise ValueError(f"{m['right']['heads']} heads are no multiple of {m['right']['kv_heads']} key heads")
                if ff is not None:
                    self.router(i)
            except ValueError as e:
                raise ValueError(f"layer {i}: {e}") from None
            if l["type"] != LATENT:
                continue
            if m["rot"]["dims"] > m["rot_dim"] or m["rot"]["dims"] % 2:
                raise ValueError(f"layer {i}: {m['rot']['dims']} rotated dimensions of {m['rot_dim']}")
            j = m.get("kv_from")
            if j is not None:
                src = self.layers[j] if 0 <= j < i else None
                if (src is None or src["type"] != LATENT or src["mixer"].get("kv_from") is not None
                        or any(src["mixer"][k] != m[k] for k in ("kv_rank", "rot_dim", "rot"))):
                    raise ValueError(f"layer {i}: kv_from must name an earlier latent layer of the same cache row")

    # what the generic engine code asks of any config
    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def num_attention_heads(self) -> int:
        return max(l["mixer"]["left"]["heads"] if l["type"] == PARALLEL else l["mixer"]["heads"] for l in self.layers)

    @property
    def num_key_value_heads(self) -> int:
        return self.num_attention_heads        # the batch packer's tile plan is not used here

    @property
    def width_pad(self) -> int:
        return gemm_k(self.hidden_size)

    @classmethod
    def from_hf(cls, d: dict) -> "MavidraConfig":
        b = d["embedding"].get("bigram")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), embedding_scale=float(d["embedding"]["scale"]),
                   norm_eps=float(d["norm"]["eps"]), layers=tuple(d["layers"]),
                   bigram=None if b is None else BigramConfig(int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])),
                   residual_mult=float(d.get("residual_mult", 1.0)),
                   max_position_embeddings=int(d.get("max_position_embeddings", 1 << 17)), raw=dict(d))

    def to_hf(self) -> dict:
        e = {"scale": self.embedding_scale}
        if self.bigram is not None:
            e["bigram"] = {"buckets": self.bigram.buckets, "mul_prev": self.bigram.mul_prev, "mul_cur": self.bigram.mul_cur}
        return {"architecture": "Mavidra", "architectures": list(self.architectures), "vocab": self.vocab_size, "width": self.hidden_size,
                "embedding": e, "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
                "layers": json.loads(json.dumps(list(self.layers)))}

    # ------------------------------------------------------------ layers
    def of_type(self, kind: str) -> tuple:
        return tuple(i for i, l in enumerate(self.layers) if l["type"] == kind)

    def attention(self, i: int) -> WindowAttentionConfig:
        """Softmax half of a parallel layer."""
        m = self.layers[i]["mixer"]["left"]
        rot = m.get("rot") or {}
        return WindowAttentionConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), int(rot.get("dims", 0)),
                                     float(rot.get("base", 1e4)), window=int((m.get("mask") or {}).get("size", 0)), sink=True, halves=True,
                                     qk_norm=True, eps=self.norm_eps, head_gate=True, out_mult=float(self.layers[i]["mixer"]["left_scale"]))

    def delta(self, i: int) -> DeltaRuleConfig:
        """Delta-rule half of a parallel layer."""
        m = self.layers[i]["mixer"]["right"]
        return DeltaRuleConfig(self.hidden_size, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], 0, 0, self.norm_eps,
                               head_decay=True, out_mult=float(self.layers[i]["mixer"]["right_scale"]))

    def latent(self, i: int) -> LatentAttentionConfig:
        m = self.layers[i]["mixer"]
        return LatentAttentionConfig(m["heads"], m["dim"], m["rot_dim"], m["rot"]["dims"], m["vdim"], m["kv_rank"], m["q_rank"],
                                     float(m["scale"]), float(m["rot"]["base"]), self.norm_eps, m.get("kv_from") is None, interleaved=True,
                                     window=int((m.get("mask") or {}).get("size", 0)), sink=False, head_gate=True)

    def gla(self, i: int, rank: int = 0) -> GatedLinearConfig:
        m = self.layers[i]["mixer"]
        return GatedLinearConfig(m["heads"], m["dim"], m["vdim"], rank, float(m["tau"]), self.norm_eps)

    def router(self, i: int) -> ScoreRouterConfig:
        r = self.layers[i]["mlp"]["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        return ScoreRouterConfig(int(r["experts"]), int(r["top"]), int(g["count"]), int(g["keep"]))

    # ------------------------------------------------------------ cache
    @property
    def head_width(self) -> int:
        return head_width(max([max(self.attention(i).dim, self.attention(i).vdim) for i in self.of_type(PARALLEL)], default=8))

    @property
    def cache_heads(self) -> int:
        return max([self.attention(i).kv_heads for i in self.of_type(PARALLEL)], default=1)

    @property
    def latent_layers(self) -> tuple:
        """Layers that store latent rows, in plane order."""
        return tuple(i for i in self.of_type(LATENT) if self.layers[i]["mixer"].get("kv_from") is None)

    def paged_specs(self) -> tuple:
        own = self.latent_layers
        return (("latent", len(own), max(self.latent(i).cache_width for i in own)),) if own else ()

    def state_specs(self) -> tuple:
        out = [] if self.bigram is None else [BIGRAM_STATE]
        for i, l in enumerate(self.layers):
            shapes = (self.gla(i).state_shapes() if l["type"] == GLA else self.delta(i).state_shapes() if l["type"] == PARALLEL else {})
            out += [(f"l{i}.{name}", shape, torch.float32) for name, shape in shapes.items()]
        return tuple(out)

    # ------------------------------------------------------------ checkpoint
    def tensor_shapes(self, ranks: Optional[dict] = None) -> dict:
        """Name -> shape of every tensor of a checkpoint. ``ranks``: rank of the decay projection per gated linear layer (not in
        the config; a checkpoint's shapes give it, 16 otherwise)."""
        W, out = self.hidden_size, {"embed": (self.vocab_size, self.hidden_size)}
        if self.bigram is not None:
            out["bigram"] = (self.bigram.buckets + 1, W)

        def norm(name):
            out.update({name: (W,), name + ".b": (W,)})

        for i, l in enumerate(self.layers):
            m, p = l["mixer"], f"l{i}.mix."
            norm(f"l{i}.norm1")
            norm(f"l{i}.norm1b")
            if l["type"] == GLA:
                H, d, dv, r = m["heads"], m["dim"], m["vdim"], (ranks or {}).get(i, 16)
                out.update({p + "q": (H * d, W), p + "k": (H * d, W), p + "v": (H * dv, W), p + "g": (H * dv, W), p + "o": (W, H * dv),
                            p + "norm": (dv,), p + "a1": (r, W), p + "a2": (H * d, r), p + "a2.b": (H * d,)})
            elif l["type"] == LATENT:
                H, d, dv = m["heads"], m["dim"], m["vdim"]
                out.update({p + "dq": (m["q_rank"], W), p + "dq.norm": (m["q_rank"],), p + "uq": (H * (d + m["rot_dim"]), m["q_rank"])})
                if m.get("kv_from") is None:
                    out.update({p + "dkv": (m["kv_rank"] + m["rot_dim"], W), p + "dkv.norm": (m["kv_rank"],)})
                out.update({p + "uk": (H * d, m["kv_rank"]), p + "uv": (H * dv, m["kv_rank"]), p + "g": (H, W), p + "o": (W, H * dv)})
            else:
                a, b, q, r = m["left"], m["right"], p + "left.", p + "right."
                H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
                out.update({q + "q": (H * d, W), q + "k": (G * d, W), q + "v": (G * dv, W), q + "q.norm": (d,), q + "k.norm": (d,),
                            q + "sink": (H,), q + "g": (H, W), q + "o": (W, H * dv)})
                H, G, d, dv = b["heads"], b["kv_heads"], b["dim"], b["vdim"]
                for n, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                    out.update({r + n: (rows, W), r + n + ".conv": (rows, b["conv"])})
                out.update({r + "b": (H, W), r + "A_log": (H,), r + "norm": (dv,), r + "a": (H, W), r + "dt_bias": (H,),
                            r + "g": (H * dv, W), r + "o": (W, H * dv)})
            ff, q = l.get("mlp"), f"l{i}.mlp."
            if ff is None:
                continue
            norm(f"l{i}.norm2")
            norm(f"l{i}.norm2b")
            F, E = ff["expert"]["ff"], ff["router"]["experts"]
            for e in range(E):
                out.update({f"{q}e{e}.gate": (F, W), f"{q}e{e}.up": (F, W), f"{q}e{e}.down": (W, F)})
            out.update({q + "router": (E, W), q + "correction": (E,)})
        norm("final.norm")
        return out

    def param_count(self) -> int:
        n = 0
        for shape in self.tensor_shapes().values():
            k = 1
            for s in shape:
                k *= s
            n += k
        return n

    @classmethod
    def build(cls, width: int, vocab: int, pattern: str, gla: dict, latent: dict, parallel: dict, expert_ff: int, router: dict,
              bigram: Optional[dict] = None, eps: float = 1e-5, embedding_scale: float = 1.0, residual_mult: float = 1.0) -> "MavidraConfig":
        """A config from a pattern of layers: ``G`` gated linear attention, ``A`` latent attention, ``S`` latent attention on the
        last A's cache rows, ``P`` the parallel mixer; a lower-case letter has no experts."""
        layers, last, copy = [], None, lambda d: json.loads(json.dumps(d))
        for i, ch in enumerate(pattern):
            kind = ch.upper()
            mixer = copy({"G": gla, "A": latent, "S": latent, "P": parallel}[kind])
            if kind == "S":
                mixer["kv_from"] = last
            elif kind == "A":
                last = i
            layers.append({"type": {"G": GLA, "P": PARALLEL}.get(kind, LATENT), "mixer": mixer,
                           "mlp": {"kind": "moe", "expert": {"ff": expert_ff}, "router": copy(router)} if ch.isupper() else None})
        b = bigram or dict(buckets=vocab, mul_prev=31, mul_cur=7)
        return cls(vocab, width, embedding_scale, eps, tuple(layers), BigramConfig(**b), residual_mult)

    @classmethod
    def tiny(cls, **kw) -> "MavidraConfig":
        base = dict(width=160, vocab=512, pattern="GAPSg", expert_ff=80, router=dict(experts=6, top=2, groups=dict(count=3, keep=2)),
                    gla=dict(heads=3, dim=24, vdim=40, tau=8.0),
                    latent=dict(heads=4, dim=40, rot_dim=24, vdim=40, kv_rank=80, q_rank=72, scale=64 ** -0.5, mask=dict(size=48),
                                rot=dict(base=10000.0, dims=24)),
                    parallel=dict(left=dict(heads=6, kv_heads=2, dim=40, vdim=48, scale=40 ** -0.5, rot=dict(base=20000.0, dims=24)),
                                  right=dict(heads=4, kv_heads=2, dim=24, vdim=32, conv=4), left_scale=0.9, right_scale=0.7),
                    bigram=dict(buckets=301, mul_prev=37, mul_cur=11), residual_mult=0.6, embedding_scale=0.8)
        base.update(kw)
        return cls.build(**base)


@dataclass
class MavidraLayer:
    norm1: tuple                                   # (weight, bias) of the layer norms
    norm1b: tuple
    mixer: object                                  # GatedLinearAttention | LatentAttention | ParallelMixer
    norm2: Optional[tuple] = None
    norm2b: Optional[tuple] = None
    router: Optional[ScoreRouter] = None
    w_gate_up: Optional[torch.Tensor] = None       # experts: [E, 2 ff, width]
    w_down: Optional[torch.Tensor] = None          # experts: [E, width, ff]


class MavidraWeights:
    def __init__(self, cfg: MavidraConfig, embed, bigram, layers, final_norm):
        self.cfg, self.embed, self.bigram, self.layers, self.final_norm = cfg, embed, bigram, layers, final_norm

    @classmethod
    def from_state_dict(cls, cfg: MavidraConfig, sd: dict, device="cpu", dtype=torch.bfloat16) -> "MavidraWeights":
        W, Wp = cfg.hidden_size, cfg.width_pad
        ranks = {i: sd[f"l{i}.mix.a1"].shape[0] for i in cfg.of_type(GLA) if f"l{i}.mix.a1" in sd}
        for name, shape in cfg.tensor_shapes(ranks).items():
            if name not in sd:
                raise KeyError(f"the checkpoint has no tensor {name!r}")
            if tuple(sd[name].shape) != tuple(shape):
                raise ValueError(f"{name}: {tuple(sd[name].shape)} in the checkpoint, {tuple(shape)} by the config")
        put = lambda t: t.to(device=device, dtype=dtype).contiguous()
        norm = lambda n: tuple(put(torch.nn.functional.pad(sd[k], (0, Wp - W))) for k in (n, n + ".b"))
        layers = []
        for i, l in enumerate(cfg.layers):
            p = f"l{i}.mix."
            t = {k[len(p):]: v for k, v in sd.items() if k.startswith(p)}
            if l["type"] == GLA:
                mixer = GatedLinearAttention(cfg.gla(i, ranks[i]), t, Wp, device, dtype)
            elif l["type"] == LATENT:
                mixer = LatentAttention(cfg.latent(i), t, Wp, device, dtype)
            else:
                side = lambda s: {k[len(s):]: v for k, v in t.items() if k.startswith(s)}
                mixer = ParallelMixer(WindowAttention(cfg.attention(i), side("left."), cfg.head_width, Wp, device, dtype),
                                      DeltaRule(cfg.delta(i), side("right."), Wp, device, dtype), device, dtype)
            lw = MavidraLayer(norm(f"l{i}.norm1"), norm(f"l{i}.norm1b"), mixer)
            ff, q = l.get("mlp"), f"l{i}.mlp."
            if ff is not None:
                E, F = ff["router"]["experts"], gemm_k(ff["expert"]["ff"])
                lw.norm2, lw.norm2b = norm(f"l{i}.norm2"), norm(f"l{i}.norm2b")
                lw.router = ScoreRouter(cfg.router(i), sd[q + "router"], sd[q + "correction"], Wp, device, dtype)
                lw.w_gate_up = put(torch.stack([torch.cat([pad_to(sd[f"{q}e{e}.{n}"], F, Wp) for n in ("gate", "up")])
                                                for e in range(E)]))
                lw.w_down = put(torch.stack([pad_to(sd[f"{q}e{e}.down"], Wp, F) for e in range(E)]))
            layers.append(lw)
        bigram = None if cfg.bigram is None else put(pad_to(sd["bigram"], cfg.bigram.buckets + 1, Wp))
        return cls(cfg, put(pad_to(sd["embed"], up8(cfg.vocab_size), Wp)), bigram, layers, norm("final.norm"))

    @staticmethod
    def random_state_dict(cfg: MavidraConfig, seed: int = 0, dtype=torch.float32, device="cpu") -> dict:
        """Random tensors of a checkpoint: projections scaled by their fan-in, norms around one, decays between slow and fast."""
        g = torch.Generator(device=device).manual_seed(seed)
        sd = {}
        for name, shape in cfg.tensor_shapes().items():
            leaf, t = name.rsplit(".", 1)[-1], torch.randn(*shape, generator=g, device=device)
            if leaf == "b" and len(shape) == 1:
                t = 1.0 + t if name.endswith("a2.b") else 0.1 * t
            elif leaf == "A_log":
                t = t.abs() - 2.0
            elif leaf == "dt_bias":
                t = t - 3.0
            elif leaf == "correction":
                t = 0.1 * t
            elif "norm" in leaf:
                t = 1.0 + 0.1 * t
            elif name not in ("embed", "bigram") and leaf != "sink":
                t = t * shape[-1] ** -0.5
            sd[name] = t.to(dtype)
        return sd

    @classmethod
    def random_init(cls, cfg: MavidraConfig, device="cpu", dtype=torch.bfloat16, seed: int = 0) -> "MavidraWeights":
        """Random weights, generated on ``device``."""
        return cls.from_state_dict(cfg, cls.random_state_dict(cfg, seed, dtype, device), device, dtype)


class MavidraModel:
    """Serves :class:`MavidraConfig` behind the engine's model interface (``forward_tensors``); decode steps replay CUDA graphs.
    ``kv_cache``: [pages, 2, parallel layers, kv heads, page, head width]; ``paged``: the cache manager's further paged tensors
    (latent rows); ``state``: its state tensors."""

    use_executor = False
    executor = None
    logits_buf = None

    def __init__(self, cfg: MavidraConfig, weights: MavidraWeights, kv_cache: torch.Tensor, max_tokens: int = 8192,
                 max_seqs: int = 256, max_position: Optional[int] = None, state: Optional[dict] = None, paged: Optional[dict] = None):
        self.cfg, self.w, self.kv, self.state, self.paged = cfg, weights, kv_cache, state or {}, paged or {}
        self.device, self.dtype = weights.embed.device, weights.embed.dtype
        self.max_tokens, self.max_seqs = max_tokens, max_seqs
        self.page_size = kv_cache.shape[4]
        self.max_position = max_position or min(cfg.max_position_embeddings, 1 << 17)
        # every attention layer's plane: among the keys and values, or among the latent rows (its own or the shared one)
        own = {i: j for j, i in enumerate(cfg.latent_layers)}
        self.plane = {i: j for j, i in enumerate(cfg.of_type(PARALLEL))}
        for i in cfg.of_type(LATENT):
            j = cfg.layers[i]["mixer"].get("kv_from")
            self.plane[i] = own[i if j is None else j]
        tables: dict = {}
        self.cos_sin = {}
        for i in self.plane:
            a = cfg.attention(i) if cfg.layers[i]["type"] == PARALLEL else cfg.latent(i)
            key = (a.rot_dims, a.rope_base)
            if key not in tables:
                tables[key] = cos_sin_table(a.rot_dims, self.max_position, a.rope_base, None, self.device) if a.rot_dims else None
            self.cos_sin[i] = tables[key]
        self.groups = sorted({cfg.attention(i).group_pad for i in cfg.of_type(PARALLEL)})
        self.moe_layers = [i for i, l in enumerate(cfg.layers) if l.get("mlp") is not None]
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
        c, w, T, Wp, dev = self.cfg, self.w, tokens.shape[0], self.cfg.width_pad, self.device
        new = lambda rows: torch.empty(rows, Wp, dtype=self.dtype, device=dev)
        seam = lambda x, **kw: sandwich_norm(x, cols=c.hidden_size, eps=c.norm_eps, **kw)
        one_token = T == q_len.shape[0]
        plans = {g: tensor_core_plan(g, self.kv.shape[5], self.dtype, self.page_size, q_start, q_len, T, one_token)
                 for g in self.groups}
        counts = torch.zeros(len(self.moe_layers), self.max_experts, dtype=torch.int32, device=dev)
        x = torch.empty(T, Wp, dtype=torch.float32, device=dev)
        # what the next seam adds to the stream: the embedding first, then one branch at a time
        pending = dict(ids=tokens, table=w.embed, scale=c.embedding_scale)
        if c.bigram is not None:
            pending.update(inject=w.bigram, inject_ids=bigram_rows(c.bigram, tokens, q_start, q_len, kv_len, state_slot,
                                                                   self.state[BIGRAM_STATE[0]]))
        routed = 0
        for i, l in enumerate(w.layers):
            h, kind = new(T), c.layers[i]["type"]
            seam(x, w1=l.norm1[0], b1=l.norm1[1], n1=h, **pending)
            if kind == GLA:
                y = l.mixer(h, ops.linear, self.state[f"l{i}.gla"], state_slot, q_start, q_len, kv_len, one_token)
            elif kind == LATENT:
                y = l.mixer(h, ops.linear, self.paged["latent"][:, self.plane[i]], self.cos_sin[i], positions, slots, block_table,
                            q_start, q_len, kv_len, one_token)
            else:
                y = l.mixer(h, ops.linear, self.kv, self.plane[i], self.state[f"l{i}.delta"], self.state[f"l{i}.conv"], self.cos_sin[i],
                            positions, slots, block_table, q_start, q_len, kv_len, state_slot, plans[l.mixer.left.cfg.group_pad],
                            one_token)
            pending = dict(a=y, w_u=l.norm1b[0], b_u=l.norm1b[1], mult=c.residual_mult)
            if l.router is not None:
                h = new(T)
                seam(x, w1=l.norm2[0], b1=l.norm2[1], n1=h, **pending)
                rows, offsets, inverse, pair_w = l.router.route(h, counts[routed, : l.router.cfg.experts])
                routed += 1
                pending = dict(e=expert_mlp(rows, offsets, l.w_gate_up, l.w_down, T), inverse=inverse, pair_w=pair_w, w_u=l.norm2b[0],
                               b_u=l.norm2b[1], mult=c.residual_mult)
            if stream is not None:
                seam(x, **pending)
                stream.append(x[:, : c.hidden_size].clone())
                pending = {}
        out = new(logit_rows.shape[0])
        if out.shape[0] == 0:
            return torch.empty(0, c.vocab_size, dtype=torch.float32, device=dev)
        seam(x, rows=logit_rows, w1=w.final_norm[0], b1=w.final_norm[1], n1=out, store_x=False, **pending)
        logits = ops.linear(out, w.embed, out_dtype=torch.float32)
        return logits if logits.shape[1] == c.vocab_size else logits[:, : c.vocab_size].contiguous()
