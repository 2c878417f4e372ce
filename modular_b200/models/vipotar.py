"""Vipotar: a decoder whose layers run windowed softmax attention, lightning attention and a feed-forward in parallel.

Every layer is ``x += m (half the sum of both mixers' normed outputs + ff)``, all three branches reading one norm of the fp32
residual stream (:mod:`modular_b200.nn.parallel_block`). A range of layers may be looped: it runs several times with the same
weights, each pass with a cache plane and a state of its own; a learned row is added to the stream before each pass, and the
embedding again before each but the first. Logits are capped softly. ``config.json`` lists the layers one by one.

Cache: a key/value plane of the paged cache and a slot of recurrent state per layer *run* (a looped layer has one for each
pass). The seam between two runs is one kernel (:func:`modular_b200.nn.residual.residual_norm`), the additions before a pass
included. Decode steps replay CUDA graphs.
"""

from __future__ import annotations

import json
import math
from dataclasses import dataclass, field
from typing import Optional

import torch

from .. import ops
from ..nn.delta_rule import gemm_k, pad_to, up8
from ..nn.lightning_attention import LightningAttention, LightningConfig
from ..nn.parallel_block import ParallelBlock
from ..nn.residual import residual_norm
from ..nn.rotary_embedding import RopeScaling, cos_sin_table
from ..nn.window_attention import WindowAttention, WindowAttentionConfig, head_width, tensor_core_plan
from .decode_graphs import DecodeGraphs


@dataclass(frozen=True)
class LayerRun:
    """One run of a layer. ``step``: the row of ``loop.step`` added before it (-1: none), with the embedding when ``inject``."""
    layer: int
    step: int = -1
    inject: bool = False


@dataclass
class VipotarConfig:
    vocab_size: int
    hidden_size: int
    rms_norm_eps: float
    layers: tuple                                   # the entries of config.json's ``layers``
    loop: Optional[dict] = None                     # {"start", "stop", "times"}
    residual_mult: float = 1.0
    logit_softcap: Optional[float] = None
    max_position_embeddings: int = 1 << 17
    architectures: tuple = ("Vipotar",)
    raw: dict = field(default_factory=dict, repr=False)

    def __post_init__(self):
        if not self.layers:
            raise ValueError("config.json lists no layers")
        for i, l in enumerate(self.layers):
            if l["type"] != "parallel":
                raise ValueError(f"layer {i}: mixer type {l['type']!r} is not known")
            if l.get("mlp") is not None and l["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {l['mlp']['kind']!r} is not known")
            try:
                self.attention(i), self.lightning(i)
            except ValueError as e:
                raise ValueError(f"layer {i}: {e}") from None
        if self.loop is not None:
            a, b, n = (int(self.loop[k]) for k in ("start", "stop", "times"))
            if not (0 <= a < b <= len(self.layers) and n >= 1):
                raise ValueError(f"loop over layers {a} .. {b - 1}, {n} times, of {len(self.layers)} layers")

    # what the generic engine code asks of any config
    @property
    def num_hidden_layers(self) -> int:
        return len(self.runs)

    @property
    def num_attention_heads(self) -> int:
        return max([l["mixer"]["left"]["heads"] for l in self.layers])

    @property
    def num_key_value_heads(self) -> int:
        return self.num_attention_heads        # the batch packer's tile plan is not used here

    @property
    def width_pad(self) -> int:
        return gemm_k(self.hidden_size)

    @classmethod
    def from_hf(cls, d: dict) -> "VipotarConfig":
        cap = d.get("logit_softcap")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), rms_norm_eps=float(d["norm"]["eps"]),
                   layers=tuple(d["layers"]), loop=d.get("loop"), residual_mult=float(d.get("residual_mult", 1.0)),
                   logit_softcap=None if cap is None else float(cap),
                   max_position_embeddings=int(d.get("max_position_embeddings", 1 << 17)), raw=dict(d))

    def to_hf(self) -> dict:
        return {"architecture": "Vipotar", "architectures": list(self.architectures), "vocab": self.vocab_size,
                "width": self.hidden_size, "norm": {"eps": self.rms_norm_eps}, "residual_mult": self.residual_mult,
                "logit_softcap": self.logit_softcap, "loop": self.loop, "layers": json.loads(json.dumps(list(self.layers)))}

    # ------------------------------------------------------------ layers
    def attention(self, i: int) -> WindowAttentionConfig:
        m = self.layers[i]["mixer"]["left"]
        rot, s = m.get("rot") or {}, (m.get("rot") or {}).get("scaling")
        scaling = None
        if s is not None:
            scaling = RopeScaling("yarn", factor=float(s["factor"]), original_max_position_embeddings=s["original"],
                                  beta_fast=float(s["fast"]), beta_slow=float(s["slow"]), attention_factor=0.1 * math.log(s["factor"]) + 1.0)
        return WindowAttentionConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), int(rot.get("dims", 0)),
                                     float(rot.get("base", 1e4)), scaling, int((m.get("mask") or {}).get("size", 0)), True)

    def lightning(self, i: int) -> LightningConfig:
        m = self.layers[i]["mixer"]["right"]
        return LightningConfig(m["heads"], m["dim"], m["vdim"], tuple(float(x) for x in m["decay"]), self.rms_norm_eps)

    @property
    def runs(self) -> tuple:
        """Layer runs in order."""
        n, loop = len(self.layers), self.loop
        if loop is None:
            return tuple(LayerRun(i) for i in range(n))
        a, b = int(loop["start"]), int(loop["stop"])
        out = [LayerRun(i) for i in range(a)]
        for t in range(int(loop["times"])):
            out += [LayerRun(a, t, t > 0)] + [LayerRun(i) for i in range(a + 1, b)]
        return tuple(out + [LayerRun(i) for i in range(b, n)])

    @property
    def head_width(self) -> int:
        return head_width(max(max(l["mixer"]["left"]["dim"], l["mixer"]["left"]["vdim"]) for l in self.layers))

    @property
    def cache_heads(self) -> int:
        return max(l["mixer"]["left"]["kv_heads"] for l in self.layers)

    def state_specs(self) -> tuple:
        return tuple((f"r{r}.{name}", shape, torch.float32) for r, run in enumerate(self.runs)
                     for name, shape in self.lightning(run.layer).state_shapes().items())

    def tensor_shapes(self) -> dict:
        """Name -> shape of every tensor of a checkpoint."""
        W, out = self.hidden_size, {"embed": (self.vocab_size, self.hidden_size)}
        if self.loop is not None:
            out["loop.step"] = (int(self.loop["times"]), W)
        for i, l in enumerate(self.layers):
            m, n, p = l["mixer"]["left"], l["mixer"]["right"], f"l{i}.mix."
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            h, e, ev = n["heads"], n["dim"], n["vdim"]
            out.update({f"l{i}.norm1": (W,), p + "left.q": (H * d, W), p + "left.k": (G * d, W), p + "left.v": (G * dv, W),
                        p + "left.o": (W, H * dv), p + "left.out": (W,), p + "right.q": (h * e, W), p + "right.k": (h * e, W),
                        p + "right.v": (h * ev, W), p + "right.g": (h * ev, W), p + "right.o": (W, h * ev),
                        p + "right.norm": (h * ev,), p + "right.out": (W,)})
            if l.get("mlp") is not None:
                F = l["mlp"]["ff"]
                out.update({f"l{i}.mlp.up": (F, W), f"l{i}.mlp.down": (W, F)})
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
    def build(cls, width: int, vocab: int, layers: int, left: dict, right: dict, ff: int, loop: Optional[dict] = None,
              eps: float = 1e-5, residual_mult: float = 1.0, logit_softcap: float = 30.0) -> "VipotarConfig":
        """A config of equal layers; ``right`` may leave out its decays (then they run from fast to slow over the heads)."""
        right = dict(right)
        right.setdefault("decay", [1.0 - 2.0 ** (-1.0 - 7.0 * h / max(right["heads"] - 1, 1)) for h in range(right["heads"])])
        entry = {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": {"kind": "dense", "ff": ff}}
        return cls(vocab, width, eps, tuple(json.loads(json.dumps(entry)) for _ in range(layers)), loop, residual_mult, logit_softcap)

    @classmethod
    def tiny(cls, **kw) -> "VipotarConfig":
        base = dict(width=160, vocab=512, layers=4, ff=224, loop={"start": 1, "stop": 3, "times": 2}, residual_mult=0.6,
                    left=dict(heads=6, kv_heads=2, dim=40, vdim=48, scale=40 ** -0.5, mask={"size": 48},
                              rot=dict(base=20000.0, dims=24, scaling=dict(factor=4.0, original=256, fast=32.0, slow=1.0))),
                    right=dict(heads=3, dim=24, vdim=40))
        base.update(kw)
        return cls.build(**base)


@dataclass
class VipotarLayer:
    norm1: torch.Tensor
    block: ParallelBlock


class VipotarWeights:
    def __init__(self, cfg: VipotarConfig, embed, layers, final_norm, head, step):
        self.cfg, self.embed, self.layers = cfg, embed, layers
        self.final_norm, self.head, self.step = final_norm, head, step

    @classmethod
    def from_state_dict(cls, cfg: VipotarConfig, sd: dict, device="cpu", dtype=torch.bfloat16) -> "VipotarWeights":
        W, Wp, V, hd = cfg.hidden_size, cfg.width_pad, cfg.vocab_size, cfg.head_width
        for name, shape in cfg.tensor_shapes().items():
            if name not in sd:
                raise KeyError(f"the checkpoint has no tensor {name!r}")
            if tuple(sd[name].shape) != tuple(shape):
                raise ValueError(f"{name}: {tuple(sd[name].shape)} in the checkpoint, {tuple(shape)} by the config")
        put = lambda t: t.to(device=device, dtype=dtype).contiguous()
        row = lambda n: put(torch.nn.functional.pad(sd[n], (0, Wp - W)))
        layers = []
        for i in range(len(cfg.layers)):
            side = lambda s: {n.rsplit(".", 1)[1]: t for n, t in sd.items() if n.startswith(f"l{i}.mix.{s}.")}
            lt, rt = side("left"), side("right")
            block = ParallelBlock(WindowAttention(cfg.attention(i), lt, hd, Wp, device, dtype),
                                  LightningAttention(cfg.lightning(i), rt, Wp, device, dtype), lt["out"], rt["out"],
                                  sd.get(f"l{i}.mlp.up"), sd.get(f"l{i}.mlp.down"), Wp, device, dtype)
            layers.append(VipotarLayer(row(f"l{i}.norm1"), block))
        step = None if cfg.loop is None else put(pad_to(sd["loop.step"], sd["loop.step"].shape[0], Wp))
        return cls(cfg, put(pad_to(sd["embed"], V, Wp)), layers, row("final.norm"), put(pad_to(sd["head"], up8(V), Wp)), step)

    @staticmethod
    def random_state_dict(cfg: VipotarConfig, seed: int = 0, dtype=torch.float32, device="cpu") -> dict:
        """Random tensors of a checkpoint: projections scaled by their fan-in, norms around one."""
        g = torch.Generator(device=device).manual_seed(seed)
        sd = {}
        for name, shape in cfg.tensor_shapes().items():
            t = torch.randn(*shape, generator=g, device=device)
            if len(shape) == 1:
                t = 1.0 + 0.1 * t
            elif name == "loop.step":
                t = 0.3 * t
            elif name != "embed":
                t = t * shape[-1] ** -0.5
            sd[name] = t.to(dtype)
        return sd

    @classmethod
    def random_init(cls, cfg: VipotarConfig, device="cpu", dtype=torch.bfloat16, seed: int = 0) -> "VipotarWeights":
        """Random weights, generated on ``device``."""
        return cls.from_state_dict(cfg, cls.random_state_dict(cfg, seed, dtype, device), device, dtype)


class VipotarModel:
    """Serves :class:`VipotarConfig` behind the engine's model interface (``forward_tensors``); decode steps replay CUDA
    graphs. ``kv_cache``: [pages, 2, layer runs, kv heads, page, head width]; ``state``: the cache manager's state tensors."""

    use_executor = False
    executor = None
    logits_buf = None

    def __init__(self, cfg: VipotarConfig, weights: VipotarWeights, kv_cache: torch.Tensor, max_tokens: int = 8192,
                 max_seqs: int = 256, max_position: Optional[int] = None, state: Optional[dict] = None):
        self.cfg, self.w, self.kv, self.state = cfg, weights, kv_cache, state or {}
        self.device, self.dtype = weights.embed.device, weights.embed.dtype
        self.max_tokens, self.max_seqs = max_tokens, max_seqs
        self.page_size, self.runs = kv_cache.shape[4], cfg.runs
        self.max_position = max_position or min(cfg.max_position_embeddings, 1 << 17)
        tables: dict = {}
        self.cos_sin = []
        for l in weights.layers:
            a = l.block.left.cfg
            key = (a.rot_dims, a.rope_base, repr(a.rope_scaling))
            if key not in tables:
                tables[key] = (cos_sin_table(a.rot_dims, self.max_position, a.rope_base, a.rope_scaling, self.device)
                               if a.rot_dims else None)
            self.cos_sin.append(tables[key])
        self.groups = sorted({l.block.left.cfg.group_pad for l in weights.layers})
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
        """``stream`` (a list) collects a copy of the residual stream after every layer run."""
        c, w, T, Wp = self.cfg, self.w, tokens.shape[0], self.cfg.width_pad
        eps, new = c.rms_norm_eps, lambda rows: torch.empty(rows, Wp, dtype=self.dtype, device=self.device)
        one_token = T == q_len.shape[0]
        plans = {g: tensor_core_plan(g, self.kv.shape[5], self.dtype, self.page_size, q_start, q_len, T, one_token)
                 for g in self.groups}
        x = torch.empty(T, Wp, dtype=torch.float32, device=self.device)
        pending = dict(ids=tokens, table=w.embed)       # what the next seam adds to the stream, the embedding first
        for r, run in enumerate(self.runs):
            l, h = w.layers[run.layer], new(T)
            if run.step >= 0:
                pending["step"] = w.step[run.step]
                if run.inject:
                    pending.update(ids=tokens, inject=w.embed)
            residual_norm(x, w1=l.norm1, n1=h, cols=c.hidden_size, eps=eps, **pending)
            pending = l.block(h, ops.linear, self.kv, r, self.state[f"r{r}.lightning"], self.cos_sin[run.layer], positions, slots,
                              block_table, q_start, q_len, kv_len, state_slot, plans[l.block.left.cfg.group_pad], one_token)
            pending["mult"] = c.residual_mult
            if stream is not None:
                residual_norm(x, cols=c.hidden_size, eps=eps, **pending)
                stream.append(x[:, : c.hidden_size].clone())
                pending = {}
        out = new(logit_rows.shape[0])
        if out.shape[0] == 0:
            return torch.empty(0, c.vocab_size, dtype=torch.float32, device=self.device)
        residual_norm(x, rows=logit_rows, w1=w.final_norm, n1=out, cols=c.hidden_size, store_x=False, eps=eps, **pending)
        logits = ops.linear(out, w.head, out_dtype=torch.float32)
        if c.logit_softcap is not None:
            ops.softcap(logits, c.logit_softcap)
        return logits if logits.shape[1] == c.vocab_size else logits[:, : c.vocab_size].contiguous()
