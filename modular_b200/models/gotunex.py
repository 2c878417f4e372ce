"""Gotunex: a decoder whose layers mix latent attention and a gated delta rule, each beside its feed-forward.

Every layer is ``x += mixer(norm1(x)) + ff(norm2(x))`` on an fp32 residual stream. The mixer is latent attention
(:mod:`modular_b200.nn.latent_attention`; a layer may read the cache rows of an earlier one) or a gated delta rule with
per-channel decay (:mod:`modular_b200.nn.delta_rule`); the feed-forward is a tanh-GELU MLP, experts chosen by token id
(:class:`modular_b200.nn.moe.TableRouter`) or absent. ``config.json`` lists the layers one by one, each with its own sizes.

Cache: one plane of the paged latent cache per layer with a key/value projection of its own; recurrent layers keep
their state in the cache manager's state slots. The seam between layers is one kernel
(:func:`modular_b200.nn.residual.residual_norm`): it adds both branches, for experts straight from expert order, and
writes the next layer's two normalised inputs, the second one in expert order when experts follow. Decode steps replay
CUDA graphs.
"""

from __future__ import annotations

import json
from dataclasses import dataclass, field
from typing import Optional

import torch

from .. import ops
from ..nn.delta_rule import DeltaRule, DeltaRuleConfig, gemm_k, pad_to, up8
from ..nn.latent_attention import LatentAttention, LatentAttentionConfig
from ..nn.moe import TableRouter, expert_mlp
from ..nn.residual import residual_norm
from ..nn.rotary_embedding import cos_sin_table
from .decode_graphs import DecodeGraphs

ATTENTION, DELTA = "latent_attention", "channel_delta"


@dataclass
class GotunexConfig:
    vocab_size: int
    hidden_size: int
    embedding_scale: float
    rms_norm_eps: float
    layers: tuple                                   # the entries of config.json's ``layers``
    max_position_embeddings: int = 1 << 17
    architectures: tuple = ("Gotunex",)
    raw: dict = field(default_factory=dict, repr=False)

    def __post_init__(self):
        if not self.layers:
            raise ValueError("config.json lists no layers")
        for i, l in enumerate(self.layers):
            m, ff = l["mixer"], l.get("mlp")
            if l["type"] not in (ATTENTION, DELTA):
                raise ValueError(f"layer {i}: mixer type {l['type']!r} is not known")
            if ff is not None and ff["kind"] not in ("dense", "moe"):
                raise ValueError(f"layer {i}: feed-forward kind {ff['kind']!r} is not known")
            if l["type"] == DELTA and m["heads"] % m["kv_heads"]:
                raise ValueError(f"layer {i}: {m['heads']} heads are no multiple of {m['kv_heads']} key heads")
            if l["type"] == ATTENTION and m["rot"]["dims"] > m["rot_dim"]:
                raise ValueError(f"layer {i}: more rotated dimensions than the rotated part has")
            j = m.get("kv_from") if l["type"] == ATTENTION else None
            if j is not None:
                src = self.layers[j] if 0 <= j < i else None
                if (src is None or src["type"] != ATTENTION or src["mixer"].get("kv_from") is not None
                        or any(src["mixer"][k] != m[k] for k in ("kv_rank", "rot_dim", "rot"))):
                    raise ValueError(f"layer {i}: kv_from must name an earlier latent layer of the same cache row")

    # what the generic engine code asks of any config
    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def num_attention_heads(self) -> int:
        return max([l["mixer"]["heads"] for l in self.layers])

    @property
    def num_key_value_heads(self) -> int:
        return self.num_attention_heads        # the batch packer's tile plan is not used here

    @property
    def width_pad(self) -> int:
        return gemm_k(self.hidden_size)

    @classmethod
    def from_hf(cls, d: dict) -> "GotunexConfig":
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), embedding_scale=float(d["embedding"]["scale"]),
                   rms_norm_eps=float(d["norm"]["eps"]), layers=tuple(d["layers"]),
                   max_position_embeddings=int(d.get("max_position_embeddings", 1 << 17)), raw=dict(d))

    def to_hf(self) -> dict:
        return {"architecture": "Gotunex", "architectures": list(self.architectures), "vocab": self.vocab_size,
                "width": self.hidden_size, "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.rms_norm_eps},
                "layers": json.loads(json.dumps(list(self.layers)))}

    # ------------------------------------------------------------ layers
    def attention(self, i: int) -> LatentAttentionConfig:
        m = self.layers[i]["mixer"]
        return LatentAttentionConfig(m["heads"], m["dim"], m["rot_dim"], m["rot"]["dims"], m["vdim"], m["kv_rank"], m["q_rank"],
                                     float(m["scale"]), float(m["rot"]["base"]), self.rms_norm_eps, m.get("kv_from") is None)

    def delta(self, i: int, decay_rank: int = 0, gate_rank: int = 0) -> DeltaRuleConfig:
        m = self.layers[i]["mixer"]
        return DeltaRuleConfig(self.hidden_size, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], decay_rank,
                               gate_rank, self.rms_norm_eps)

    def is_attention(self, i: int) -> bool:
        return self.layers[i]["type"] == ATTENTION

    def mlp_kind(self, i: int) -> Optional[str]:
        ff = self.layers[i].get("mlp")
        return None if ff is None else ff["kind"]

    @property
    def cache_layers(self) -> tuple:
        """Layers that store rows in the latent cache, in plane order."""
        return tuple(i for i, l in enumerate(self.layers) if l["type"] == ATTENTION and l["mixer"].get("kv_from") is None)

    @property
    def cache_width(self) -> int:
        return max([self.attention(i).cache_width for i in self.cache_layers], default=8)

    @property
    def recurrent_layers(self) -> tuple:
        return tuple(i for i, l in enumerate(self.layers) if l["type"] == DELTA)

    def state_specs(self) -> tuple:
        return tuple((f"l{i}.{name}", shape, torch.float32) for i in self.recurrent_layers
                     for name, shape in self.delta(i).state_shapes().items())

    def tensor_shapes(self) -> dict:
        """Name -> shape of every tensor of a checkpoint. The ranks of the low-rank decay and gate projections are not in
        the config (a checkpoint's shapes give them); here they are the key width."""
        W, out = self.hidden_size, {"embed": (self.vocab_size, self.hidden_size)}
        for i, l in enumerate(self.layers):
            m, p = l["mixer"], f"l{i}.mix."
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            out[f"l{i}.norm1"] = (W,)
            if l["type"] == ATTENTION:
                out.update({p + "dq": (m["q_rank"], W), p + "dq.norm": (m["q_rank"],), p + "uq": (H * (d + m["rot_dim"]), m["q_rank"])})
                if m.get("kv_from") is None:
                    out.update({p + "dkv": (m["kv_rank"] + m["rot_dim"], W), p + "dkv.norm": (m["kv_rank"],)})
                out.update({p + "uk": (H * d, m["kv_rank"]), p + "uv": (H * dv, m["kv_rank"]), p + "sink": (H,),
                            p + "g": (H * dv, W), p + "o": (W, H * dv)})
            else:
                kd = m["kv_heads"] * d
                for n, rows in (("q", kd), ("k", kd), ("v", H * dv)):
                    out.update({p + n: (rows, W), p + n + ".conv": (rows, m["conv"])})
                out.update({p + "b": (H, W), p + "A_log": (H,), p + "dt_bias": (H * d,), p + "norm": (dv,), p + "a1": (d, W),
                            p + "a2": (H * d, d), p + "g1": (d, W), p + "g2": (H * dv, d), p + "o": (W, H * dv)})
            ff, q = l.get("mlp"), f"l{i}.mlp."
            if ff is None:
                continue
            out[f"l{i}.norm2"] = (W,)
            if ff["kind"] == "dense":
                out.update({q + "up": (ff["ff"], W), q + "down": (W, ff["ff"])})
            else:
                F = ff["expert"]["ff"]
                for e in range(ff["router"]["experts"]):
                    out.update({f"{q}e{e}.gate": (F, W), f"{q}e{e}.up": (F, W), f"{q}e{e}.down": (W, F)})
                out[q + "table"] = (self.vocab_size, ff["router"]["top"])
        out.update({"final.norm": (W,), "head": (self.vocab_size, W)})
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
    def build(cls, width: int, vocab: int, pattern: str, attention: dict, delta: dict, dense_ff: int, expert_ff: int,
              experts: int, top: int, eps: float = 1e-5, embedding_scale: float = 1.0) -> "GotunexConfig":
        """A config from a pattern of layers: ``A`` latent attention, ``S`` latent attention on the last A's cache rows,
        ``D`` delta rule; a lower-case letter has a dense feed-forward, an upper-case one experts."""
        layers, last = [], None
        for i, ch in enumerate(pattern):
            kind = ch.upper()
            if kind == "D":
                mixer, t = dict(delta), DELTA
            else:
                mixer, t = json.loads(json.dumps(attention)), ATTENTION
                if kind == "S":
                    mixer["kv_from"] = last
                else:
                    last = i
            ff = ({"kind": "dense", "ff": dense_ff} if ch.islower() else
                  {"kind": "moe", "expert": {"ff": expert_ff}, "router": {"experts": experts, "top": top}})
            layers.append({"type": t, "mixer": mixer, "mlp": ff})
        return cls(vocab, width, embedding_scale, eps, tuple(layers))

    @classmethod
    def tiny(cls, **kw) -> "GotunexConfig":
        base = dict(width=192, vocab=512, pattern="dASdD", dense_ff=320, expert_ff=96, experts=6, top=2,
                    attention=dict(heads=4, dim=48, rot_dim=24, vdim=40, kv_rank=96, q_rank=72, scale=72 ** -0.5,
                                   rot=dict(base=10000.0, dims=24)),
                    delta=dict(heads=4, kv_heads=2, dim=40, vdim=24, conv=4))
        base.update(kw)
        return cls.build(**base)


@dataclass
class GotunexLayer:
    norm1: torch.Tensor
    mixer: object                                  # LatentAttention | DeltaRule
    norm2: Optional[torch.Tensor] = None
    w_up: Optional[torch.Tensor] = None            # dense: [ff, width], [width, ff]
    w_down: Optional[torch.Tensor] = None          # experts: [E, width, ff]
    w_gate_up: Optional[torch.Tensor] = None       # experts: [E, 2 ff, width]
    moe_index: int = -1                            # position among the layers with experts


class GotunexWeights:
    def __init__(self, cfg: GotunexConfig, embed, layers, final_norm, head, router: TableRouter):
        self.cfg, self.embed, self.layers = cfg, embed, layers
        self.final_norm, self.head, self.router = final_norm, head, router

    @classmethod
    def from_state_dict(cls, cfg: GotunexConfig, sd: dict, device="cpu", dtype=torch.bfloat16) -> "GotunexWeights":
        W, Wp = cfg.hidden_size, cfg.width_pad
        put = lambda t: t.to(device=device, dtype=dtype).contiguous()
        row = lambda n: put(torch.nn.functional.pad(sd[n], (0, Wp - W)))
        layers, tables, experts = [], [], []
        for i, l in enumerate(cfg.layers):
            p = f"l{i}.mix."
            t = {k[len(p):]: v for k, v in sd.items() if k.startswith(p)}
            if cfg.is_attention(i):
                mixer = LatentAttention(cfg.attention(i), t, Wp, device, dtype)
            else:
                mixer = DeltaRule(cfg.delta(i, t["a1"].shape[0], t["g1"].shape[0]), t, Wp, device, dtype)
            lw = GotunexLayer(row(f"l{i}.norm1"), mixer)
            ff, q = l.get("mlp"), f"l{i}.mlp."
            if ff is not None:
                lw.norm2 = row(f"l{i}.norm2")
            if ff is not None and ff["kind"] == "dense":
                F = gemm_k(ff["ff"])
                lw.w_up, lw.w_down = put(pad_to(sd[q + "up"], F, Wp)), put(pad_to(sd[q + "down"], Wp, F))
            elif ff is not None:
                E, F = ff["router"]["experts"], gemm_k(ff["expert"]["ff"])
                lw.w_gate_up = put(torch.stack([torch.cat([pad_to(sd[f"{q}e{e}.{n}"], F, Wp) for n in ("gate", "up")])
                                                for e in range(E)]))
                lw.w_down = put(torch.stack([pad_to(sd[f"{q}e{e}.down"], Wp, F) for e in range(E)]))
                lw.moe_index = len(tables)
                tables.append(sd[q + "table"])
                experts.append(E)
            layers.append(lw)
        return cls(cfg, put(pad_to(sd["embed"], cfg.vocab_size, Wp)), layers, row("final.norm"),
                   put(pad_to(sd["head"], up8(cfg.vocab_size), Wp)), TableRouter(tables, experts, device))

    @staticmethod
    def random_state_dict(cfg: GotunexConfig, seed: int = 0, dtype=torch.float32, device="cpu") -> dict:
        """Random tensors of a checkpoint: projections scaled by their fan-in, norms around one, decays between slow and
        fast, a table with distinct experts per row."""
        g = torch.Generator(device=device).manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, generator=g, device=device)
        sd = {}
        for name, shape in cfg.tensor_shapes().items():
            leaf = name.rsplit(".", 1)[-1]
            if leaf == "table":
                E = cfg.layers[int(name.split(".")[0][1:])]["mlp"]["router"]["experts"]
                sd[name] = torch.rand(shape[0], E, generator=g, device=device).topk(shape[1], dim=-1).indices.int()
                continue
            if leaf == "A_log":
                t = torch.rand(*shape, generator=g, device=device) * 2.0 - 2.0
            elif leaf == "dt_bias":
                t = rnd(*shape) - 3.0
            elif leaf == "sink":
                t = rnd(*shape)
            elif "norm" in leaf:
                t = 1.0 + 0.1 * rnd(*shape)
            elif leaf == "conv":
                t = rnd(*shape) * shape[-1] ** -0.5
            elif name == "embed":
                t = rnd(*shape)
            else:
                t = rnd(*shape) * shape[-1] ** -0.5
            sd[name] = t.to(dtype)
        return sd

    @classmethod
    def random_init(cls, cfg: GotunexConfig, device="cpu", dtype=torch.bfloat16, seed: int = 0) -> "GotunexWeights":
        """Random weights, generated on ``device``."""
        return cls.from_state_dict(cfg, cls.random_state_dict(cfg, seed, dtype, device), device, dtype)


class GotunexModel:
    """Serves :class:`GotunexConfig` behind the engine's model interface (``forward_tensors``); decode steps replay CUDA
    graphs. ``kv_cache``: [pages, 1, cache layers, 1, page, cache width]; ``state``: the cache manager's state tensors."""

    use_executor = False
    executor = None
    logits_buf = None

    def __init__(self, cfg: GotunexConfig, weights: GotunexWeights, kv_cache: torch.Tensor, max_tokens: int = 8192,
                 max_seqs: int = 256, max_position: Optional[int] = None, state: Optional[dict] = None):
        self.cfg, self.w, self.kv, self.state = cfg, weights, kv_cache, state or {}
        self.device, self.dtype = weights.embed.device, weights.embed.dtype
        self.max_tokens, self.max_seqs = max_tokens, max_seqs
        self.page_size = kv_cache.shape[4]
        plane = {i: j for j, i in enumerate(cfg.cache_layers)}
        # every latent layer's cache plane: its own, or the one of the layer it reads from
        self.plane = {i: plane[l["mixer"].get("kv_from", i) if l["mixer"].get("kv_from") is not None else i]
                      for i, l in enumerate(cfg.layers) if cfg.is_attention(i)}
        max_position = max_position or min(cfg.max_position_embeddings, 1 << 17)
        tables: dict = {}
        self.cos_sin = {}
        for i in self.plane:
            a = cfg.attention(i)
            key = (a.rot_dims, a.rope_base)
            if key not in tables:
                tables[key] = cos_sin_table(a.rot_dims, max_position, a.rope_base, None, self.device)
            self.cos_sin[i] = tables[key]
        self.graphs: Optional[DecodeGraphs] = None
        self.forward_calls = 0

    # ------------------------------------------------------------ CUDA graphs of decode steps
    def capture_decode_graphs(self, batch_sizes) -> None:
        if self.device.type != "cuda":
            return
        if self.graphs is None:
            longest = max([t.shape[0] for t in self.cos_sin.values()], default=1 << 17)
            self.graphs = DecodeGraphs(self._forward, self.device,
                                       -(-min(longest, self.kv.shape[0] * self.page_size) // self.page_size), self.max_seqs)
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
        c, w, T, Wp = self.cfg, self.w, tokens.shape[0], self.cfg.width_pad
        dev, eps = self.device, self.cfg.rms_norm_eps
        new = lambda rows: torch.empty(rows, Wp, dtype=self.dtype, device=dev)
        # the tiled GEMM for every step size: the decode-step GEMM measured 2 to 29 % slower per step at these widths
        lin = ops.linear
        one_token = T == q_len.shape[0]
        routes = w.router.route(tokens)
        x = torch.empty(T, Wp, dtype=torch.float32, device=dev)
        # what the next seam adds to the stream: the embedding first, then both branches of a layer
        pending = dict(ids=tokens, table=w.embed, scale=c.embedding_scale)
        for i, l in enumerate(w.layers):
            n1, n2, inverse, offsets = new(T), None, None, None
            if l.norm2 is not None:
                if l.moe_index >= 0:
                    inverse, offsets = routes[l.moe_index]
                n2 = new(T if inverse is None else inverse.numel())
            residual_norm(x, w1=l.norm1, n1=n1, w2=l.norm2, n2=n2, scatter=inverse, cols=c.hidden_size, eps=eps, **pending)
            if c.is_attention(i):
                y = l.mixer(n1, lin, self.kv[:, 0, self.plane[i], 0], self.cos_sin[i], positions, slots, block_table, q_start,
                            q_len, kv_len, one_token)
            else:
                y = l.mixer(n1, lin, self.state[f"l{i}.delta"], self.state[f"l{i}.conv"], state_slot, q_start, q_len, kv_len,
                            one_token)
            pending = dict(a=y)
            if inverse is not None:
                e = expert_mlp(n2, offsets, l.w_gate_up, l.w_down, T)
                pending.update(e=e, inverse=inverse, pair_w=1.0 / inverse.shape[1])
            elif n2 is not None:
                pending.update(b=lin(ops.gelu_tanh(lin(n2, l.w_up)), l.w_down))
            if stream is not None:
                residual_norm(x, **pending)
                stream.append(x[:, : c.hidden_size].clone())
                pending = {}
        out = new(logit_rows.shape[0])
        if out.shape[0] == 0:
            return torch.empty(0, c.vocab_size, dtype=torch.float32, device=dev)
        residual_norm(x, rows=logit_rows, w1=w.final_norm, n1=out, cols=c.hidden_size, store_x=False, eps=eps, **pending)
        logits = ops.linear(out, w.head, out_dtype=torch.float32)
        return logits if logits.shape[1] == c.vocab_size else logits[:, : c.vocab_size].contiguous()
