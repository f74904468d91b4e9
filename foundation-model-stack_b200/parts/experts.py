"""Routed feed-forwards: many small experts, of which every token uses a few.

``RoutedExperts`` ("routed_experts").  With h the feed-forward's input:

    s = sigmoid(Wr h)                         router scores, float32
    the ``top`` experts with the largest scores are the token's; their scores are its weights, as they are
    expert_e(v) = Wdown,e (g * sigmoid(alpha g) * (u + 1)),  g = min(Wgate,e v, limit),  u = clamp(Wup,e v, -limit, limit)
    y = sum over the chosen e of expert_e(s_e * h)        the weight multiplies the expert's INPUT

The experts' matrices are stacked: ``gate_up`` [experts, 2 hidden, dim] (gate rows, then up rows) and ``down``
[experts, dim, hidden].  A step sorts its (token, choice) pairs by expert on the device (no answer from the device is
waited for), runs the two products group by group with the gated unit in the first one's epilogue, and sums every
token's rows.  Options of the ``FeedForwardSpec``: ``experts``, ``top``, ``limit``, ``alpha`` (1.702).

Further options, each of which leaves the above as it is when absent:

    ``scoring`` "softmax"     s = softmax(Wr h) over all experts; a token's experts are the ``top`` largest of
                              s + ``correction`` (a vector of the checkpoint, one number an expert, where ``correction``
                              is set); its weights are the chosen scores s (without the correction) over their sum
                              (+ 1e-20), times ``route_scale``; the weight multiplies the expert's OUTPUT
    ``scoring`` "sigmoid_groups"  s = sigmoid(Wr h); the choice is by s + ``correction``, and the experts form ``groups``
                              equal groups of neighbours of which the ``keep`` best can be chosen from (a group's score:
                              the sum of its two largest choice scores); the weights are the chosen s as they are, times
                              ``route_scale``, and multiply the experts' OUTPUTS
    ``scoring`` "softmax_chosen"  the ``top`` largest logits Wr h + ``router_bias`` (a vector of the checkpoint, where
                              ``router_bias`` is set) are a token's experts, its weights the softmax over those logits
                              alone, times ``route_scale``; they multiply the experts' OUTPUTS
    ``unit`` "relu_squared"   expert_e(v) = Wdown,e relu(Wup,e v)^2: no gate; ``up`` [experts, hidden, dim]
    ``unit`` "silu"           expert_e(v) = Wdown,e (silu(Wgate,e v) * Wup,e v)
    ``shared`` spec           a further unit that runs for every token: a ``projected_unit``, whose products the block makes
                              with its mixer's, or a feed-forward of its own, whose output is added here
    ``shared_gate``           the latter's output is multiplied by sigmoid(w h), one number a token; w is the row of the
                              router's matrix behind the experts' rows (the router's product makes both; ``router_rows``)
"""
from __future__ import annotations

import torch

from ..config.specs import FeedForwardSpec
from ..kernels import ops
from .base import Part
from .linear import Linear
from .registry import build_feed_forward, register_feed_forward


class RoutedExperts(Part):
    _ROUTE_MODES = {"sigmoid": ops.ROUTE_SIGMOID, "softmax": ops.ROUTE_SOFTMAX, "sigmoid_groups": ops.ROUTE_SIGMOID_GROUPS,
                    "softmax_chosen": ops.ROUTE_SOFTMAX_CHOSEN}

    def __init__(self, spec: FeedForwardSpec) -> None:
        super().__init__()
        o = dict(spec.options)
        self.experts, self.top = int(o["experts"]), int(o["top"])
        self.limit, self.alpha = float(o.get("limit", 0.0)), float(o.get("alpha", 1.702))
        self.hidden = int(spec.hidden)
        if not (0 < self.top <= self.experts) or self.hidden <= 0:
            raise ValueError(f"routed_experts: {self.experts} experts, top {self.top}, hidden {self.hidden}")
        self.scoring, self.unit = o.get("scoring", "sigmoid"), o.get("unit", "gated_clamped")
        if self.scoring not in self._ROUTE_MODES or self.unit not in ("gated_clamped", "relu_squared", "silu"):
            raise ValueError(f"routed_experts: scoring {self.scoring!r}, unit {self.unit!r}")
        if self.unit == "gated_clamped" and "limit" not in o:
            raise ValueError("routed_experts: the gated unit needs its limit")
        self.route_scale, self.has_correction = float(o.get("route_scale", 1.0)), bool(o.get("correction", False))
        self.groups, self.keep = int(o.get("groups", 1)), int(o.get("keep", 1))
        if (self.groups <= 0 or self.experts % self.groups or not (0 < self.keep <= self.groups)
                or self.keep * (self.experts // self.groups) < self.top):
            raise ValueError(f"routed_experts: {self.experts} experts in {self.groups} groups of which {self.keep} stay, "
                             f"top {self.top}")
        shared = build_feed_forward(o["shared"]) if o.get("shared") is not None else None
        self.shared = None
        if shared is not None and not hasattr(shared, "in_rows"):  # a feed-forward with products of its own
            self.shared, shared = self.add("shared", shared), None
        self.shared_gate = bool(o.get("shared_gate", False))
        if self.shared_gate and self.shared is None:
            raise ValueError("routed_experts: a gate without a shared unit of its own")
        self.in_rows = shared.in_rows if shared else 0
        self.joint_hidden, self.activation = (shared.hidden, shared.activation) if shared else (0, 0)
        self.gated = shared.gated if shared else False
        self.router = self.add("router", Linear(spec.dim, self.router_rows(self.experts, self.shared_gate), False))
        self.has_bias = bool(o.get("router_bias", False))
        if self.has_bias:
            self.declare("router_bias", (self.experts,), role="vector")
        if self.has_correction:
            self.declare("correction", (self.experts,), role="vector")
        if self.unit == "relu_squared":
            self.declare("up", (self.experts, self.hidden, spec.dim), role="matrix")
        else:
            self.declare("gate_up", (self.experts, 2 * self.hidden, spec.dim), role="matrix")
        self.declare("down", (self.experts, spec.dim, self.hidden), role="matrix")
        self._correction = self._bias = None

    @staticmethod
    def router_rows(experts: int, shared_gate: bool) -> int:
        """Rows of the router's matrix: what a checkpoint adapter has to put together ([router; shared gate; zeros up to a
        multiple of 8, so that the library's product finds its rows aligned])."""
        return (experts + 1 + 7) // 8 * 8 if shared_gate else experts

    def finalize(self, device, dtype) -> None:
        super().finalize(device, dtype)
        if self.has_correction:
            self._correction = self.tensor("correction").float().contiguous()
        if self.has_bias:
            self._bias = self.tensor("router_bias").float().contiguous()

    def beside(self, x):
        """What a block that makes its sublayers' products together adds as it is: the routed experts."""
        return self._routed(x)

    def forward(self, x):
        if self.in_rows:
            raise ValueError("routed_experts: a shared unit belongs to a block that makes its products (parallel_joint)")
        return self._routed(x)

    def _routed(self, x):
        every = self.shared.forward(x) if self.shared is not None else None
        mode, further = self._ROUTE_MODES[self.scoring], {"bias": self._bias, "side": self.shared_gate, "experts": self.experts}
        if self.scoring == "sigmoid":
            routing = ops.route(x, self.router.tensor("weight"), self.top, mode, **further)
        else:
            routing = ops.route(x, self.router.tensor("weight"), self.top, mode, self._correction, self.route_scale, self.groups,
                                self.keep, **further)
        if self.unit == "relu_squared":
            hidden = ops.routed_linear(routing.rows, self.tensor("up"), routing, relu_squared=True)
            return ops.route_gather(ops.routed_linear(hidden, self.tensor("down"), routing), routing, every)
        hidden = ops.routed_linear(routing.rows, self.tensor("gate_up"), routing, True, self.limit, self.alpha,
                                   silu=self.unit == "silu")
        return ops.route_gather(ops.routed_linear(hidden, self.tensor("down"), routing), routing, every)

    def kernel_libraries(self, dtype):
        own = self.shared.kernel_libraries(dtype) if self.shared is not None else []
        return own + ["grouped", "elementwise"] + (["gemm_bf16_skinny"] if dtype == torch.bfloat16 else [])


register_feed_forward("routed_experts", RoutedExperts)
