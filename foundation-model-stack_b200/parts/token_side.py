"""What a layer adds for the tokens themselves, after its sublayers.

``TokenSide``: with x the stream after the layer's sublayers and e the token's row of the layer's own table,

    y = Wproj (act(Wgate x) * e);   x += y / sqrt(mean(y^2) + eps) * norm

``gate`` [dim, width] and ``proj`` [width, dim] are small matrices (dim values a token and layer), the table
[vocabulary, dim] is the layer's.  The sum x += the sublayers' outputs and the copy of x in the compute dtype that Wgate
reads come from one kernel; y stays pending with its norm, for whichever norm comes next.
"""
from __future__ import annotations

import torch

from ..config.specs import NormSpec, TokenSideSpec
from ..kernels import ops
from .base import Part
from .feedforward import UNGATED_ACTIVATIONS
from .linear import Linear
from .norm import NormedDelta
from .registry import build_norm


class TokenSide(Part):
    def __init__(self, spec: TokenSideSpec) -> None:
        super().__init__()
        if spec.dim <= 0 or spec.vocab_size <= 0 or spec.activation not in UNGATED_ACTIVATIONS:
            raise ValueError(f"token side: {spec.dim} values of {spec.vocab_size} tokens, activation {spec.activation!r}")
        self.activation = UNGATED_ACTIVATIONS[spec.activation]
        self.declare("table", (spec.vocab_size, spec.dim), role="matrix")
        self.gate = self.add("gate", Linear(spec.width, spec.dim))
        self.proj = self.add("proj", Linear(spec.dim, spec.width))
        self.norm = self.add("norm", build_norm(NormSpec("rmsnorm", spec.width, spec.eps)))

    def forward(self, residual, parts, batch, dtype):
        """``parts``: the sublayers' outputs with their factors, which the stream does not hold yet."""
        if dtype == torch.float32:
            ops.normed_add_norm(residual, parts, None, None, dtype, want_out=False)
            x = residual
        else:
            x = ops.normed_add_norm(residual, parts, None, None, dtype)
        g = ops.token_gated_linear(x, self.gate.tensor("weight"), self.tensor("table"), batch.tokens, self.activation)
        return NormedDelta(self.proj.forward(g), self.norm)

    def kernel_libraries(self, dtype):
        return super().kernel_libraries(dtype) + ["elementwise"]
