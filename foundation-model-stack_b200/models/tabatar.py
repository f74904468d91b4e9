"""Tabatar: a decoder with several residual streams a token (hyper-connections), pre-norm layers whose mixer is either
grouped-query attention (queries and keys normed per head, then turned in halves; a window; a sigmoid gate a value) or gated
linear attention (a matrix memory per head with one decay a key channel), each followed by an ungated feed-forward
(gelu), by routed experts beside a gated shared one (weights: the softmax over the chosen logits alone), or by nothing.  A
run of layers may be passed through several times with the same weights, every pass with a cache or state of its own.  The
logits are scaled, then capped by a tanh.

This file is all that is specific to the architecture: its ``config.json`` (``vocab``, ``width``, ``norm.eps``,
``embedding.scale``, ``streams``, ``loop`` {start, stop, times} or null, ``logit_scale``, ``logit_softcap``, and ``layers``,
each entry with its ``type``, the sizes and constants of its ``mixer`` and its ``mlp`` or null), the ``DecoderSpec`` that
configuration means, and the checkpoint's tensor names:

    embed [vocab, width]   final.norm [width]   head [vocab, width]   l<i>.norm1, l<i>.norm2 [width]
    l<i>.hc1, .hc2:  .in, .out [streams], .mix [streams, streams] (from, to)
    attention: l<i>.mix.q, .k, .v, .g, .o, .q.norm, .k.norm [dim]
    gla:       l<i>.mix.q, .k, .v, .g, .o, .norm [vdim], .a1 [rank, width], .a2 [heads * dim, rank], .a2.b
    dense:     l<i>.mlp.up [ff, width], .down [width, ff]
    experts:   l<i>.mlp.router [experts, width], .router.b, .e<j>.gate, .up [ff, width], .e<j>.down [width, ff],
               .shared.gate, .up, .down, .shared.sg [1, width]

Linear weights are stored [out, in].  The rank of a decay is not in config.json: it is read from the shape of ``a1``.  The
adapter makes one matrix of [q; k; v; g] and of [q; k; v; g; a1] (filled up with zero rows to a multiple of 8), of
[gate; up], of [router; sg], and stacks the experts.  A layer that runs again is a further entry of the decoder's layers
with the earlier one's weights.
"""
from __future__ import annotations

import copy
import dataclasses
import re
from typing import Any, Dict, List, Optional

import torch

from ..config.model_config import ModelConfig
from ..config.specs import BlockSpec, DecoderSpec, FeedForwardSpec, LayerCall, MixerSpec, NormSpec, PositionSpec
from ..parts.experts import RoutedExperts
from ..parts.linear_attention import GatedLinearAttention
from ..weights.adapters import register_adapter, register_adapter_step
from ..weights.sources import TensorLayout
from . import register_architecture, register_model
from .base import Model

LAYER_TYPES = ("attention", "gla")
MLP_KINDS = ("dense", "moe")


@dataclasses.dataclass
class TabatarConfig(ModelConfig):
    vocab: int = 512
    width: int = 256
    norm_eps: float = 1e-6
    embedding_scale: float = 1.0
    streams: int = 2  # 0: one residual stream, to which the sublayers add
    logit_scale: float = 1.0
    logit_softcap: float = 0.0  # 0: no cap
    loop: Optional[Dict[str, int]] = None  # {"start", "stop", "times"}
    layers: List[Dict[str, Any]] = dataclasses.field(default_factory=list)
    max_positions: int = 131072  # how long a sequence may get; nothing in the model depends on it

    def __post_init__(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or self.streams < 0:
            raise ValueError(f"vocab {self.vocab}, width {self.width}, {self.streams} streams")
        for i, layer in enumerate(self.layers):
            if layer.get("type") not in LAYER_TYPES:
                raise ValueError(f"layer {i}: type {layer.get('type')!r}; known: {', '.join(LAYER_TYPES)}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind") not in MLP_KINDS:
                raise ValueError(f"layer {i}: feed-forward kind {mlp.get('kind')!r}; known: {', '.join(MLP_KINDS)}, or null")
        if self.loop is not None:
            a, b, n = (int(self.loop[k]) for k in ("start", "stop", "times"))
            if not (0 <= a <= b <= len(self.layers)) or n < 1:
                raise ValueError(f"loop {self.loop} over {len(self.layers)} layers")

    def order(self) -> List[int]:
        """The layers in the order in which they run."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b, times = (int(self.loop[k]) for k in ("start", "stop", "times"))
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))


def _config_from_json(values: Dict[str, Any]) -> TabatarConfig:
    if values.get("architecture") != "Tabatar":
        raise ValueError(f"config.json is of architecture {values.get('architecture')!r}, not Tabatar")
    absent = [k for k in ("vocab", "width", "layers", "norm") if k not in values]
    if absent:
        raise ValueError(f"config.json lacks {absent}")

    def number(value, default: float) -> float:
        return default if value is None else float(value)

    return TabatarConfig(vocab=int(values["vocab"]), width=int(values["width"]), norm_eps=float(values["norm"]["eps"]),
                         embedding_scale=number((values.get("embedding") or {}).get("scale"), 1.0),
                         streams=int(values.get("streams") or 0), logit_scale=number(values.get("logit_scale"), 1.0),
                         logit_softcap=number(values.get("logit_softcap"), 0.0), loop=copy.deepcopy(values.get("loop")) or None,
                         layers=copy.deepcopy(values["layers"]), max_positions=int(values.get("max_positions", 131072)))


# ---- layer entries as config.json has them -----------------------------------------------------------
def dense_mlp(ff: int) -> dict:
    return {"kind": "dense", "ff": ff}


def moe_mlp(experts: int, top: int, ff: int, shared_ff: int = 0) -> dict:
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared_ff:
        out["shared"] = {"ff": shared_ff}
    return out


def attention_layer(heads: int, kv_heads: int, dim: int, vdim: int, scale: float, window: int, rot: Optional[dict],
                    mlp: Optional[dict]) -> dict:
    mixer = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if window:
        mixer["mask"] = {"size": window}
    if rot:
        mixer["rot"] = copy.deepcopy(rot)
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def gla_layer(heads: int, dim: int, vdim: int, tau: float, rank: int, mlp: Optional[dict]) -> dict:
    return {"type": "gla", "mixer": {"dim": dim, "heads": heads, "tau": tau, "vdim": vdim, "rank": rank}, "mlp": mlp}


def _sizes(mixer: dict):
    """(heads, key/value heads, size of queries and keys, size of values)."""
    h, d = int(mixer["heads"]), int(mixer["dim"])
    return h, int(mixer.get("kv_heads") or h), d, int(mixer.get("vdim") or d)


def _window(mixer: dict) -> int:
    return int((mixer.get("mask") or {}).get("size") or 0)


def _shared_ff(mlp: dict) -> int:
    return int((mlp.get("shared") or {}).get("ff") or 0)


class Tabatar(Model):
    architecture = "tabatar"
    default_source = "native"

    def __init__(self, config: Optional[TabatarConfig] = None, **kwargs) -> None:
        config = config if config is not None else TabatarConfig()
        super().__init__(config.updated(**kwargs))

    @classmethod
    def config_from_json(cls, values: dict) -> TabatarConfig:
        return _config_from_json(values)

    def config_json(self) -> dict:
        c = self.config
        return {"architecture": "Tabatar", "vocab": c.vocab, "width": c.width, "norm": {"eps": c.norm_eps},
                "embedding": {"scale": c.embedding_scale}, "streams": c.streams, "loop": copy.deepcopy(c.loop),
                "logit_scale": c.logit_scale, "logit_softcap": c.logit_softcap, "layers": copy.deepcopy(c.layers)}

    def load(self, source, adapter_source, device, dtype):
        # what config.json leaves out is read from the checkpoint's names and shapes
        names = set(source.keys())

        def fill(target: dict, key: str, name: str, axis: int = 0) -> None:
            if target.get(key) is None and name in names:
                target[key] = int(source.spec(name)[1][axis])

        c = self.config
        connected = next((n for n in sorted(names) if n.endswith(".hc1.in")), None)
        if connected is None and c.streams == 1:
            c.streams = 0  # one stream without weights of its own: plain sums
        elif connected is not None and not c.streams:
            c.streams = int(source.spec(connected)[1][0])
        for i, layer in enumerate(c.layers):
            if layer["type"] == "gla":
                fill(layer["mixer"], "rank", f"l{i}.mix.a1")
            mlp, p = layer.get("mlp"), f"l{i}.mlp."
            if mlp is None:
                continue
            if mlp["kind"] == "dense":
                fill(mlp, "ff", p + "up")
                continue
            fill(mlp.setdefault("expert", {}), "ff", p + "e0.up")
            fill(mlp.setdefault("router", {}), "experts", p + "router")
            if mlp.get("shared") is not None or p + "shared.up" in names:
                if mlp.get("shared") is None:
                    mlp["shared"] = {}
                fill(mlp["shared"], "ff", p + "shared.up")
        return super().load(source, adapter_source, device, dtype)

    # ---- specs -------------------------------------------------------------------------------
    def _mixer_spec(self, layer: dict) -> MixerSpec:
        m, eps = layer["mixer"], float(self.config.norm_eps)
        h, g, d, v = _sizes(m)
        if layer["type"] == "gla":
            return MixerSpec("gla", dim=self.config.width, nheads=h, head_dim=d,
                             options=(("vdim", v), ("eps", eps), ("tau", float(m["tau"])), ("rank", int(m.get("rank") or 0))))
        rot = m.get("rot") or {}
        scaling, position = rot.get("scaling"), PositionSpec("none")
        if int(rot.get("dims") or 0):
            position = PositionSpec(
                "rope", head_dim=int(rot["dims"]), theta=float(rot["base"]),
                scaling=() if not scaling else (("rope_type", "llama3"), ("factor", float(scaling["factor"])),
                                                ("low_freq_factor", float(scaling["low"])),
                                                ("high_freq_factor", float(scaling["high"])),
                                                ("original_max_position_embeddings", float(scaling["original"]))))
        return MixerSpec("sink_attention", dim=self.config.width, nheads=h, kvheads=g, head_dim=d, window=_window(m),
                         scale=float(m["scale"]) if m.get("scale") is not None else None, position=position,
                         options=(("vdim", v), ("rot_dims", int(rot.get("dims") or 0)), ("pairing", "halves"),
                                  ("qk_norm", "before"), ("eps", eps), ("gate", True)))

    def _feed_forward_spec(self, mlp: Optional[dict]) -> Optional[FeedForwardSpec]:
        d = self.config.width
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return FeedForwardSpec("mlp", dim=d, hidden=int(mlp["ff"]), activation="gelu-tanh")
        shared = FeedForwardSpec("glu", dim=d, hidden=_shared_ff(mlp), activation="silu") if _shared_ff(mlp) else None
        return FeedForwardSpec("routed_experts", dim=d, hidden=int(mlp["expert"]["ff"]),
                               options=(("experts", int(mlp["router"]["experts"])), ("top", int(mlp["router"]["top"])),
                                        ("scoring", "softmax_chosen"), ("router_bias", True), ("unit", "silu"), ("shared", shared),
                                        ("shared_gate", shared is not None)))

    def decoder_spec(self) -> DecoderSpec:
        c = self.config
        norm = NormSpec("rmsnorm", c.width, float(c.norm_eps))
        arrangement, options = ("hyper_connected", (("streams", int(c.streams)),)) if c.streams else ("pre_norm", ())
        blocks: List[BlockSpec] = []
        for layer in c.layers:
            ff = self._feed_forward_spec(layer.get("mlp"))
            blocks.append(BlockSpec(mixer=self._mixer_spec(layer), feed_forward=ff, mixer_norm=norm,
                                    feed_forward_norm=norm if ff is not None else None, arrangement=arrangement,
                                    names=("norm1", "mix", "norm2", "mlp"), options=options))
        # a layer's first run is its own entry; every further one an entry with that layer's weights
        schedule, seen = [], set()
        for i in c.order():
            if i in seen:
                blocks.append(dataclasses.replace(blocks[i], weights_of=i))
                schedule.append(LayerCall(len(blocks) - 1))
            else:
                seen.add(i)
                schedule.append(LayerCall(i))
        return DecoderSpec(vocab_size=c.vocab, dim=c.width, layers=tuple(blocks), schedule=tuple(schedule), final_norm=norm,
                           tie_head=False, max_positions=int(c.max_positions),
                           names=("embedding", "layers", "final_norm", "head"), embedding_scale=float(c.embedding_scale),
                           logit_scale=float(c.logit_scale), logit_softcap=float(c.logit_softcap), streams=int(c.streams))

    def checkpoint_layout(self) -> List[TensorLayout]:
        c = self.config
        d, s = c.width, int(c.streams)
        out = [TensorLayout("embed", (c.vocab, d), "embedding")]
        for i, layer in enumerate(c.layers):
            p, mlp = f"l{i}.", layer.get("mlp")
            h, g, k, v = _sizes(layer["mixer"])
            for q in (1, 2) if mlp is not None else (1,):
                out.append(TensorLayout(p + f"norm{q}", (d,), "gain"))
                if s:
                    out += [TensorLayout(p + f"hc{q}.in", (s,), "gain"), TensorLayout(p + f"hc{q}.out", (s,), "gain"),
                            TensorLayout(p + f"hc{q}.mix", (s, s), "around_zero")]
            if layer["type"] == "gla":
                r = int(layer["mixer"].get("rank") or 0)
                out += [TensorLayout(p + "mix.q", (h * k, d), "matrix"), TensorLayout(p + "mix.k", (h * k, d), "matrix"),
                        TensorLayout(p + "mix.norm", (v,), "gain"), TensorLayout(p + "mix.a1", (r, d), "matrix"),
                        TensorLayout(p + "mix.a2", (h * k, r), "matrix"), TensorLayout(p + "mix.a2.b", (h * k,), "gain"),
                        TensorLayout(p + "mix.v", (h * v, d), "matrix")]
            else:
                out += [TensorLayout(p + "mix.q", (h * k, d), "matrix"), TensorLayout(p + "mix.k", (g * k, d), "matrix"),
                        TensorLayout(p + "mix.q.norm", (k,), "gain"), TensorLayout(p + "mix.k.norm", (k,), "gain"),
                        TensorLayout(p + "mix.v", (g * v, d), "matrix")]
            out += [TensorLayout(p + "mix.g", (h * v, d), "matrix"), TensorLayout(p + "mix.o", (d, h * v), "matrix")]
            if mlp is not None and mlp["kind"] == "dense":
                f = int(mlp["ff"])
                out += [TensorLayout(p + "mlp.up", (f, d), "matrix"), TensorLayout(p + "mlp.down", (d, f), "matrix")]
            elif mlp is not None:
                n = int(mlp["router"]["experts"])
                out += [TensorLayout(p + "mlp.router", (n, d), "matrix"), TensorLayout(p + "mlp.router.b", (n,), "around_zero")]
                units = [(f"e{j}", int(mlp["expert"]["ff"])) for j in range(n)]
                if _shared_ff(mlp):
                    units.append(("shared", _shared_ff(mlp)))
                    out.append(TensorLayout(p + "mlp.shared.sg", (1, d), "matrix"))
                for name, f in units:
                    out += [TensorLayout(p + f"mlp.{name}.gate", (f, d), "matrix"), TensorLayout(p + f"mlp.{name}.up", (f, d), "matrix"),
                            TensorLayout(p + f"mlp.{name}.down", (d, f), "matrix")]
        out += [TensorLayout("final.norm", (d,), "gain"), TensorLayout("head", (c.vocab, d), "head")]
        return out


# ---- checkpoint adapter ------------------------------------------------------------------------------
_LAYER = re.compile(r"^l(\d+)\.(.*)$")
_EXPERT = re.compile(r"^mlp\.e(\d+)\.(gate|up|down)$")
_RENAMED = {  # checkpoint name within a layer -> the engine's
    "norm1": "norm1.weight", "norm2": "norm2.weight", "mix.o": "mix.dense.weight", "mix.q.norm": "mix.q_norm",
    "mix.k.norm": "mix.k_norm", "mix.norm": "mix.norm", "mix.a2": "mix.decay_out.weight", "mix.a2.b": "mix.decay_out.bias",
    "mlp.up": "mlp.w1.weight", "mlp.shared.down": "mlp.shared.w2.weight", "mlp.router.b": "mlp.router_bias",
}
_RENAMED.update({f"hc{q}.{n}": f"hc{q}.{n}" for q in (1, 2) for n in ("in", "out", "mix")})


def _fuse(held: Dict[str, torch.Tensor], names, out: Dict[str, torch.Tensor], target: str, rows: int = 0) -> bool:
    """Concatenates the tensors ``names`` of ``held`` along their rows, filled up with zeros to ``rows``, into out[target] if
    all of them are there and agree in their width."""
    if not all(n in held for n in names) or len({held[n].shape[1:] for n in names}) != 1:
        return False
    parts = [held.pop(n) for n in names]
    have = sum(t.shape[0] for t in parts)
    if rows > have:
        parts.append(torch.zeros((rows - have,) + tuple(parts[0].shape[1:]), dtype=parts[0].dtype, device=parts[0].device))
    out[target] = torch.cat(parts, dim=0)
    return True


def _native_to_engine(tensors: Dict[str, torch.Tensor], config: TabatarConfig = None, **_) -> Dict[str, torch.Tensor]:
    """Names and layouts of the checkpoint -> the engine's.  Incomplete sets (a projection without its partners) are
    passed on under their own names, so that the loader's one error lists them."""
    out: Dict[str, torch.Tensor] = {}
    layers: Dict[int, Dict[str, torch.Tensor]] = {}
    top = {"embed": "embedding.weight", "final.norm": "final_norm.weight", "head": "head.weight"}
    for name, t in tensors.items():
        m = _LAYER.match(name)
        if m:
            layers.setdefault(int(m.group(1)), {})[m.group(2)] = t
        else:
            out[top.get(name, name)] = t
    for i, held in layers.items():
        p = f"layers.{i}."
        layer = config.layers[i] if config is not None and i < len(config.layers) else {}
        mlp = layer.get("mlp") or {}
        joint = ["mix.q", "mix.k", "mix.v", "mix.g"]
        if layer.get("type") == "gla":
            h, _, k, v = _sizes(layer["mixer"])
            rank = held["mix.a1"].shape[0] if "mix.a1" in held else 0
            _fuse(held, joint + ["mix.a1"], out, p + "mix.in_proj.weight", GatedLinearAttention.fused_rows(h, k, v, rank))
        else:
            _fuse(held, joint, out, p + "mix.in_proj.weight")
        if mlp.get("kind") == "moe":
            n, gate = int(mlp["router"].get("experts") or 0), bool(_shared_ff(mlp))
            _fuse(held, ["mlp.router"] + (["mlp.shared.sg"] if gate else []), out, p + "mlp.router.weight",
                  RoutedExperts.router_rows(n, gate))
            _fuse(held, ["mlp.shared.gate", "mlp.shared.up"], out, p + "mlp.shared.wg1_fused.weight")
            experts: Dict[int, Dict[str, torch.Tensor]] = {}
            for k in list(held):
                m = _EXPERT.match(k)
                if m:
                    experts.setdefault(int(m.group(1)), {})[m.group(2)] = held[k]
            n = len(experts)
            if n and sorted(experts) == list(range(n)) and all(len(e) == 3 for e in experts.values()):
                out[p + "mlp.gate_up"] = torch.stack([torch.cat([experts[j]["gate"], experts[j]["up"]]) for j in range(n)])
                out[p + "mlp.down"] = torch.stack([experts[j]["down"] for j in range(n)])
                for j in range(n):
                    for kind in ("gate", "up", "down"):
                        del held[f"mlp.e{j}.{kind}"]
        elif "mlp.down" in held:
            out[p + "mlp.w2.weight"] = held.pop("mlp.down")
        for k in list(held):
            if k in _RENAMED:
                out[p + _RENAMED[k]] = held.pop(k)
        for k, t in held.items():  # whatever found no place keeps its name and is reported
            out[f"l{i}.{k}"] = t
    return out


register_architecture("tabatar", Tabatar, config_json_names=("Tabatar",))
register_adapter_step("tabatar", "native_to_engine", _native_to_engine)
register_adapter("tabatar", "native", ["native_to_engine"])


# ---- variants ----------------------------------------------------------------------------------------
def mixed(n_layers: int, width: int, vocab: int, streams: int, heads: int, kv_heads: int, dim: int, vdim: int, window: int,
          gla_heads: int, gla_dim: int, gla_vdim: int, rank: int, ff: int, experts: int, top: int, expert_ff: int,
          shared_ff: int, loop: Optional[dict]) -> TabatarConfig:
    """Layers that take turns: attention with a dense feed-forward, gated linear attention with experts."""
    rot = {"base": 500000.0, "dims": dim, "scaling": {"factor": 8.0, "high": 4.0, "low": 1.0, "original": 8192}}
    kinds = [attention_layer(heads, kv_heads, dim, vdim, dim ** -0.5, window, rot, dense_mlp(ff)),
             gla_layer(gla_heads, gla_dim, gla_vdim, 16.0, rank, moe_mlp(experts, top, expert_ff, shared_ff))]
    return TabatarConfig(vocab=vocab, width=width, embedding_scale=width ** 0.5, streams=streams, logit_scale=1.0, logit_softcap=30.0,
                         loop=loop, layers=[copy.deepcopy(kinds[i % 2]) for i in range(n_layers)])


def _factory(config: TabatarConfig):
    def make(**kwargs) -> Tabatar:
        return Tabatar(copy.deepcopy(config), **kwargs)

    return make


# "tiny": for trying things out.  "8b-shape": layers of the width of the Llama-3-8B benchmark (4,096 wide, two streams; 32
# heads of 128 over 8 with a window of 4,096; memories of 32 heads of 128 x 128; a dense feed-forward of 14,336 or 16 experts
# of 3,584 of which a token takes 4 beside a shared one of 3,584), with which the two are measured side by side.
register_model("tabatar", "tiny", _factory(mixed(4, 64, 256, 3, 4, 2, 16, 24, 40, 2, 16, 24, 8, 96, 8, 2, 48, 32,
                                                 {"start": 1, "stop": 3, "times": 2})))
register_model("tabatar", "8b-shape", _factory(mixed(30, 4096, 128256, 2, 32, 8, 128, 128, 4096, 32, 128, 128, 16, 14336, 16, 4,
                                                     3584, 3584, None)))
