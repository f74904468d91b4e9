"""Feed-forwards.  ``GatedLinearUnit``: y = W2 (act(Wg x) * (W1 x)) with the gate and up rows fused into
one matrix, gate first (fms/modules/feedforward.py:227-240 for the sizes, :288-297 for the formula).

``PlainUnit`` ("mlp"): y = W2 act(W1 x), ungated.

Interface of a feed-forward (what a block calls):

    forward(x) -> y          x, y: [tokens, dim] in the compute dtype

A feed-forward with routing implements the same call and keeps router and experts inside.

``ProjectedUnit`` ("projected_unit"): the hidden values of a feed-forward whose two products a block makes together with
its mixer's (``JointParallelBlock``): act(up) of ``hidden`` columns, or, option ``gated``, act(gate) * up of twice as many.
It has no tensors; what such a block asks of a feed-forward is

    in_rows, joint_hidden, activation, gated       rows of the joint projection and what becomes of them
    beside(x) -> y or None                         what it computes from the block's normed input by itself (routed experts)
"""
from __future__ import annotations

from ..config.specs import FeedForwardSpec
from ..kernels import ops
from .base import Part
from .linear import Linear
from .registry import register_feed_forward

ACTIVATIONS = {"silu": 0, "swish": 0, "gelu": 1, "gelu-tanh": 2, "gelu_pytorch_tanh": 2, "relu": 3}
# for the kernels of ``ops.joint_activation`` and ``ops.token_gate``, which also know the square of relu
UNGATED_ACTIVATIONS = dict(ACTIVATIONS, relu_squared=4)


class GatedLinearUnit(Part):
    def __init__(self, spec: FeedForwardSpec) -> None:
        super().__init__()
        act = spec.activation.lower()
        if act not in ACTIVATIONS:
            raise ValueError(f"activation {spec.activation!r} is not supported; supported: {sorted(ACTIVATIONS)}")
        self.activation = ACTIVATIONS[act]
        self.hidden = spec.hidden
        self.gate_up = self.add("wg1_fused", Linear(spec.dim, 2 * spec.hidden, spec.bias))
        self.down = self.add("w2", Linear(spec.hidden, spec.dim, spec.bias))

    def forward(self, x):
        h = ops.gated_linear(x, self.gate_up.tensor("weight"), self.gate_up.tensor("bias"), self.activation)
        return self.down.forward(h)

    def kernel_libraries(self, dtype):
        return super().kernel_libraries(dtype) + ["elementwise"]


class PlainUnit(Part):
    def __init__(self, spec: FeedForwardSpec) -> None:
        super().__init__()
        act = spec.activation.lower()
        if act not in UNGATED_ACTIVATIONS:
            raise ValueError(f"activation {spec.activation!r} is not supported; supported: {sorted(UNGATED_ACTIVATIONS)}")
        self.activation = UNGATED_ACTIVATIONS[act]
        self.up = self.add("w1", Linear(spec.dim, spec.hidden, spec.bias))
        self.down = self.add("w2", Linear(spec.hidden, spec.dim, spec.bias))

    def forward(self, x):
        return self.down.forward(ops.activated_linear(x, self.up.tensor("weight"), self.up.tensor("bias"), self.activation))

    def kernel_libraries(self, dtype):
        return super().kernel_libraries(dtype) + ["elementwise"]


class ProjectedUnit(Part):
    def __init__(self, spec: FeedForwardSpec) -> None:
        super().__init__()
        act = spec.activation.lower()
        if act not in UNGATED_ACTIVATIONS:
            raise ValueError(f"activation {spec.activation!r} is not supported; supported: {sorted(UNGATED_ACTIVATIONS)}")
        if spec.bias or spec.hidden <= 0:
            raise ValueError(f"projected_unit: {spec.hidden} hidden values, bias {spec.bias}")
        self.activation, self.hidden = UNGATED_ACTIVATIONS[act], int(spec.hidden)
        self.joint_hidden = self.hidden
        self.gated = bool(dict(spec.options).get("gated", False))
        self.in_rows = self.hidden * (2 if self.gated else 1)

    def beside(self, x):
        return None


register_feed_forward("glu", GatedLinearUnit)
register_feed_forward("mlp", PlainUnit)
register_feed_forward("projected_unit", ProjectedUnit)
