"""Bolinex: a decoder with learned positions whose layers run mixer and feed-forward side by side on ONE layer norm,
x += mixer(h) + mlp(h) with h = norm1(x), and then add something of the tokens' own:
x += rms(Wproj (gelu(Wgate x) * e)) * w, e being the layer's part of the token's row of a side table.

The mixer is grouped-query attention without rotation: scores q.k * scale, capped by a tanh, less
r1_h ln(1 + r2_h * distance), over the last ``mask.size`` keys; the layers that say ``v_mix`` mix their values with those
of the first such layer (v = (1 - vmix) v + vmix v_first, before they are cached); a sigmoid gate on the heads' results.
The feed-forward is dense (Wdown relu(Wup h)^2), or routed experts with a shared one beside them (scores sigmoid(z), the
choice by score + correction within the ``groups.keep`` best of ``groups.count`` groups, weights the scores as they are,
experts Wdown (silu(Wgate h) * Wup h)), or none (null).

This file is all that is specific to the architecture: its ``config.json`` (``vocab``, ``width``, ``norm.eps``,
``max_positions``, ``token_side.dim``, and ``layers``, each entry with its ``type``, the sizes and constants of its
``mixer`` and its ``mlp`` or null), the ``DecoderSpec`` that configuration means, and the checkpoint's tensor names:

    embed [vocab, width]   pos [max_positions, width]   side.embed [vocab, layers * dim]   head [vocab, width]
    final.norm, final.norm.b, l<i>.norm1, l<i>.norm1.b [width]
    l<i>.mix.q, .k, .v, .g, .o, .r1, .r2 [heads], .vmix [] (where v_mix)
    dense:   l<i>.mlp.up [ff, width], .down [width, ff]
    experts: l<i>.mlp.router [experts, width], .correction [experts], .e<j>.gate, .up [ff, width], .e<j>.down [width, ff],
             .shared.gate, .up [ff, width], .shared.down [width, ff]
    l<i>.side.gate [dim, width], .side.proj [width, dim], .side.norm [width]

Linear weights are stored [out, in].  The adapter makes a layer's two joint matrices, [q; k; v; g; up] (with experts:
[q; k; v; g; shared gate; shared up]) and [o | down], stacks the experts as [gate; up] and down, and cuts the side table
into one table a layer.
"""
from __future__ import annotations

import copy
import dataclasses
import re
from typing import Any, Dict, List, Optional

import torch

from ..config.model_config import ModelConfig
from ..config.specs import (BlockSpec, DecoderSpec, EmbeddingSpec, FeedForwardSpec, LayerCall, MixerSpec, NormSpec,
                            TokenSideSpec)
from ..weights.adapters import register_adapter, register_adapter_step
from ..weights.sources import TensorLayout
from . import register_architecture, register_model
from .base import Model

LAYER_TYPES = ("attention",)
MLP_KINDS = ("dense", "moe")


@dataclasses.dataclass
class BolinexConfig(ModelConfig):
    vocab: int = 512
    width: int = 256
    norm_eps: float = 1e-6
    side_dim: int = 0  # values of a token's own row a layer; 0: the layers add nothing of the kind
    max_positions: int = 2048
    layers: List[Dict[str, Any]] = dataclasses.field(default_factory=list)

    def __post_init__(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or self.max_positions <= 0 or self.side_dim < 0:
            raise ValueError(f"vocab {self.vocab}, width {self.width}, {self.max_positions} positions, side {self.side_dim}")
        for i, layer in enumerate(self.layers):
            if layer.get("type") not in LAYER_TYPES:
                raise ValueError(f"layer {i}: type {layer.get('type')!r}; known: {', '.join(LAYER_TYPES)}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind") not in MLP_KINDS:
                raise ValueError(f"layer {i}: feed-forward kind {mlp.get('kind')!r}; known: {', '.join(MLP_KINDS)}, or null")

    def first_mixing_layer(self) -> Optional[int]:
        """The layer whose values the later layers that say v_mix mix theirs with."""
        return next((i for i, layer in enumerate(self.layers) if layer["mixer"].get("v_mix")), None)


def _config_from_json(values: Dict[str, Any]) -> BolinexConfig:
    if values.get("architecture") != "Bolinex":
        raise ValueError(f"config.json is of architecture {values.get('architecture')!r}, not Bolinex")
    absent = [k for k in ("vocab", "width", "layers", "norm", "max_positions") if k not in values]
    if absent:
        raise ValueError(f"config.json lacks {absent}")
    return BolinexConfig(vocab=int(values["vocab"]), width=int(values["width"]), norm_eps=float(values["norm"]["eps"]),
                         side_dim=int((values.get("token_side") or {}).get("dim", 0)),
                         max_positions=int(values["max_positions"]), layers=copy.deepcopy(values["layers"]))


# ---- layer entries as config.json has them -----------------------------------------------------------
def dense_mlp(ff: int) -> dict:
    return {"kind": "dense", "ff": ff}


def moe_mlp(experts: int, top: int, ff: int, shared_ff: int, groups: int, keep: int) -> dict:
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}},
            "shared": {"ff": shared_ff}}


def attention_layer(heads: int, kv_heads: int, dim: int, vdim: int, scale: float, softcap: float, window: int, v_mix: bool,
                    mlp: Optional[dict]) -> dict:
    return {"type": "attention", "mlp": mlp,
            "mixer": {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": window}, "scale": scale,
                      "softcap": softcap, "v_mix": v_mix, "vdim": vdim}}


def _sizes(mixer: dict):
    """(heads, key/value heads, size of queries and keys, size of values)."""
    h, d = int(mixer["heads"]), int(mixer["dim"])
    return h, int(mixer.get("kv_heads") or h), d, int(mixer.get("vdim") or d)


def _shared_ff(mlp: dict) -> int:
    return int((mlp.get("shared") or {}).get("ff", 0))


class Bolinex(Model):
    architecture = "bolinex"
    default_source = "native"

    def __init__(self, config: Optional[BolinexConfig] = None, **kwargs) -> None:
        config = config if config is not None else BolinexConfig()
        super().__init__(config.updated(**kwargs))

    @classmethod
    def config_from_json(cls, values: dict) -> BolinexConfig:
        return _config_from_json(values)

    def config_json(self) -> dict:
        c = self.config
        out = {"architecture": "Bolinex", "vocab": c.vocab, "width": c.width, "norm": {"eps": c.norm_eps},
               "max_positions": c.max_positions, "layers": copy.deepcopy(c.layers)}
        if c.side_dim:
            out["token_side"] = {"dim": c.side_dim}
        return out

    def load(self, source, adapter_source, device, dtype):
        # a size that config.json leaves out is read from the checkpoint's shapes
        names = set(source.keys())

        def fill(target: dict, key: str, name: str, axis: int = 0) -> None:
            if target.get(key) is None and name in names:
                target[key] = int(source.spec(name)[1][axis])

        for i, layer in enumerate(self.config.layers):
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            p = f"l{i}.mlp."
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
    def _mixer_spec(self, i: int, layer: dict) -> MixerSpec:
        m = layer["mixer"]
        h, g, d, v = _sizes(m)
        mixing = "" if not m.get("v_mix") else ("first" if i == self.config.first_mixing_layer() else "mixed")
        return MixerSpec("sink_attention", dim=self.config.width, nheads=h, kvheads=g, head_dim=d, scale=float(m["scale"]),
                         window=int((m.get("mask") or {}).get("size") or 0),
                         options=(("vdim", v), ("gate", True), ("softcap", float(m.get("softcap") or 0.0)), ("distance", True),
                                  ("v_mix", mixing), ("projections", "outside")))

    def _feed_forward_spec(self, mlp: Optional[dict]) -> Optional[FeedForwardSpec]:
        d = self.config.width
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return FeedForwardSpec("projected_unit", dim=d, hidden=int(mlp["ff"]), activation="relu_squared")
        r = mlp["router"]
        groups = r.get("groups") or {"count": 1, "keep": 1}
        shared = None
        if _shared_ff(mlp):
            shared = FeedForwardSpec("projected_unit", dim=d, hidden=_shared_ff(mlp), activation="silu", options=(("gated", True),))
        return FeedForwardSpec("routed_experts", dim=d, hidden=int(mlp["expert"]["ff"]),
                               options=(("experts", int(r["experts"])), ("top", int(r["top"])), ("scoring", "sigmoid_groups"),
                                        ("correction", True), ("groups", int(groups["count"])), ("keep", int(groups["keep"])),
                                        ("unit", "silu"), ("shared", shared)))

    def decoder_spec(self) -> DecoderSpec:
        c = self.config
        norm = NormSpec("layernorm", c.width, float(c.norm_eps), options=(("bias", True),))
        side = TokenSideSpec(c.vocab, c.side_dim, c.width, float(c.norm_eps)) if c.side_dim else None
        blocks = [BlockSpec(mixer=self._mixer_spec(i, layer), feed_forward=self._feed_forward_spec(layer.get("mlp")),
                            mixer_norm=norm, feed_forward_norm=None, arrangement="parallel_joint",
                            names=("norm1", "mix", "", "mlp"), token_side=side) for i, layer in enumerate(c.layers)]
        return DecoderSpec(vocab_size=c.vocab, dim=c.width, layers=tuple(blocks),
                           schedule=tuple(LayerCall(i) for i in range(len(blocks))), final_norm=norm, tie_head=False,
                           max_positions=int(c.max_positions), names=("embedding", "layers", "final_norm", "head"),
                           embedding=EmbeddingSpec("table_and_positions", (("positions", int(c.max_positions)),)))

    def checkpoint_layout(self) -> List[TensorLayout]:
        c = self.config
        d = c.width
        out = [TensorLayout("embed", (c.vocab, d), "embedding"), TensorLayout("pos", (c.max_positions, d), "embedding")]
        if c.side_dim:
            out.append(TensorLayout("side.embed", (c.vocab, len(c.layers) * c.side_dim), "embedding"))
        for i, layer in enumerate(c.layers):
            p = f"l{i}."
            h, g, k, v = _sizes(layer["mixer"])
            out += [TensorLayout(p + "norm1", (d,), "gain"), TensorLayout(p + "norm1.b", (d,), "around_zero"),
                    TensorLayout(p + "mix.q", (h * k, d), "matrix"), TensorLayout(p + "mix.k", (g * k, d), "matrix"),
                    TensorLayout(p + "mix.v", (g * v, d), "matrix"), TensorLayout(p + "mix.g", (h * v, d), "matrix"),
                    TensorLayout(p + "mix.r1", (h,), "gain"), TensorLayout(p + "mix.r2", (h,), "gain"),
                    TensorLayout(p + "mix.o", (d, h * v), "matrix")]
            if layer["mixer"].get("v_mix"):
                out.append(TensorLayout(p + "mix.vmix", (), "around_zero"))
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] == "dense":
                f = int(mlp["ff"])
                out += [TensorLayout(p + "mlp.up", (f, d), "matrix"), TensorLayout(p + "mlp.down", (d, f), "matrix")]
            elif mlp is not None:
                n, units = int(mlp["router"]["experts"]), []
                out += [TensorLayout(p + "mlp.router", (n, d), "matrix"), TensorLayout(p + "mlp.correction", (n,), "around_zero")]
                units = [(f"e{j}", int(mlp["expert"]["ff"])) for j in range(n)]
                if _shared_ff(mlp):
                    units.append(("shared", _shared_ff(mlp)))
                for name, f in units:
                    out += [TensorLayout(p + f"mlp.{name}.gate", (f, d), "matrix"), TensorLayout(p + f"mlp.{name}.up", (f, d), "matrix"),
                            TensorLayout(p + f"mlp.{name}.down", (d, f), "matrix")]
            if c.side_dim:
                out += [TensorLayout(p + "side.gate", (c.side_dim, d), "matrix"), TensorLayout(p + "side.proj", (d, c.side_dim), "matrix"),
                        TensorLayout(p + "side.norm", (d,), "gain")]
        out += [TensorLayout("final.norm", (d,), "gain"), TensorLayout("final.norm.b", (d,), "around_zero"),
                TensorLayout("head", (c.vocab, d), "head")]
        return out


# ---- checkpoint adapter ------------------------------------------------------------------------------
_LAYER = re.compile(r"^l(\d+)\.(.*)$")
_EXPERT = re.compile(r"^mlp\.e(\d+)\.(gate|up|down)$")
_RENAMED = {  # checkpoint name within a layer -> the engine's
    "norm1": "norm1.weight", "norm1.b": "norm1.bias", "mix.r1": "mix.r1", "mix.r2": "mix.r2", "mix.vmix": "mix.vmix",
    "mlp.router": "mlp.router.weight", "mlp.correction": "mlp.correction",
    "side.gate": "side.gate.weight", "side.proj": "side.proj.weight", "side.norm": "side.norm.weight",
}


def _native_to_engine(tensors: Dict[str, torch.Tensor], config: BolinexConfig = None, **_) -> Dict[str, torch.Tensor]:
    """Names and layouts of the checkpoint -> the engine's.  Incomplete sets (a projection without its partners) are
    passed on under their own names, so that the loader's one error lists them."""
    out: Dict[str, torch.Tensor] = {}
    layers: Dict[int, Dict[str, torch.Tensor]] = {}
    top = {"embed": "embedding.weight", "pos": "embedding.positions", "final.norm": "final_norm.weight",
           "final.norm.b": "final_norm.bias", "head": "head.weight"}
    n_layers = len(config.layers) if config is not None else 0
    for name, t in tensors.items():
        m = _LAYER.match(name)
        if m:
            layers.setdefault(int(m.group(1)), {})[m.group(2)] = t
        elif name == "side.embed" and n_layers and config.side_dim and t.shape[1] == n_layers * config.side_dim:
            for i in range(n_layers):  # every layer's own columns
                out[f"layers.{i}.side.table"] = t[:, i * config.side_dim:(i + 1) * config.side_dim]
        else:
            out[top.get(name, name)] = t
    for i, held in layers.items():
        p = f"layers.{i}."
        mlp = (config.layers[i].get("mlp") if config is not None and i < n_layers else None) or {}
        into, outof = ["mix.q", "mix.k", "mix.v", "mix.g"], ["mix.o"]
        if mlp.get("kind") == "dense":
            into, outof = into + ["mlp.up"], outof + ["mlp.down"]
        elif mlp and _shared_ff(mlp):
            into, outof = into + ["mlp.shared.gate", "mlp.shared.up"], outof + ["mlp.shared.down"]
        for names, axis, target in ((into, 0, "in_proj.weight"), (outof, 1, "out_proj.weight")):
            if all(n in held for n in names) and len({held[n].shape[1 - axis] for n in names}) == 1:
                out[p + target] = torch.cat([held.pop(n) for n in names], dim=axis)
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
        for k in list(held):
            if k in _RENAMED:
                out[p + _RENAMED[k]] = held.pop(k)
        for k, t in held.items():  # whatever found no place keeps its name and is reported
            out[f"l{i}.{k}"] = t
    return out


register_architecture("bolinex", Bolinex, config_json_names=("Bolinex",))
register_adapter_step("bolinex", "native_to_engine", _native_to_engine)
register_adapter("bolinex", "native", ["native_to_engine"])


# ---- variants ----------------------------------------------------------------------------------------
def mixed(n_layers: int, width: int, vocab: int, max_positions: int, heads: int, kv_heads: int, dim: int, vdim: int,
          window: int, ff: int, experts: int, top: int, groups: int, keep: int, expert_ff: int, shared_ff: int,
          side_dim: int) -> BolinexConfig:
    """Layers that take turns: a dense feed-forward, then routed experts with a shared one."""
    kinds = [dense_mlp(ff), moe_mlp(experts, top, expert_ff, shared_ff, groups, keep)]
    layers = [attention_layer(heads, kv_heads, dim, vdim, dim ** -0.5, 30.0, window, True, kinds[i % 2]) for i in range(n_layers)]
    return BolinexConfig(vocab=vocab, width=width, side_dim=side_dim, max_positions=max_positions, layers=copy.deepcopy(layers))


def _factory(config: BolinexConfig):
    def make(**kwargs) -> Bolinex:
        return Bolinex(copy.deepcopy(config), **kwargs)

    return make


# "tiny": for trying things out.  "8b-shape": layers of the width of the Llama-3-8B benchmark (4,096 wide; 32 heads of 128
# over 8; a window of 4,096; a dense feed-forward of 14,336 or 16 experts of 3,584 of which a token takes 4, in four groups
# of which two are kept, and a shared one of 3,584; 256 values a token and layer at the side), with which the two are
# measured side by side.
register_model("bolinex", "tiny", _factory(mixed(4, 64, 256, 512, 4, 2, 16, 24, 40, 96, 8, 2, 4, 2, 48, 32, 8)))
register_model("bolinex", "8b-shape", _factory(mixed(30, 4096, 128256, 8192, 32, 8, 128, 128, 4096, 14336, 16, 4, 4, 2, 3584,
                                                     3584, 256)))
