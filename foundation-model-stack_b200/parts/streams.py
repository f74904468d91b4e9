"""Several residual streams a token instead of one (hyper-connections).  All streams start as the token's embedding; a
sublayer reads a weighted sum of them and its output goes into every one of them, while they are mixed among themselves:

    u = sum_s in_s X_s;   y = sublayer(norm(u));   X_t <- sum_s mix[s, t] X_s + out_t y       all streams at once
    after the last layer the streams are summed

``HyperConnection`` holds one sublayer's ``in`` [streams], ``out`` [streams] and ``mix`` [streams, streams] (from, to).
``StreamSet`` is what the decoder hands from layer to layer in the place of the one residual stream: float32
[tokens, streams, dim], or still the embedding's rows [tokens, dim] where no sublayer has written yet (all streams are
equal then, and the first sublayer's output is what makes them differ).  ``StreamMix`` is a sublayer's output on its way
into the streams: the kernel that norms the next sublayer's input (or the decoder's last sum) mixes it in on the way.
"""
from __future__ import annotations

import torch

from .base import Part

MAX_STREAMS = 16


class StreamSet:
    __slots__ = ("start", "rows", "streams")

    def __init__(self, start: torch.Tensor, streams: int) -> None:
        self.start = start  # [tokens, dim]: every stream's rows until ``rows`` is there
        self.rows = None  # [tokens, streams, dim]
        self.streams = int(streams)


class HyperConnection(Part):
    def __init__(self, streams: int) -> None:
        super().__init__()
        if not 1 <= streams <= MAX_STREAMS:
            raise ValueError(f"hyper-connections: {streams} streams (1 to {MAX_STREAMS})")
        self.streams = int(streams)
        self.declare("in", (self.streams,), role="vector")
        self.declare("out", (self.streams,), role="vector")
        self.declare("mix", (self.streams, self.streams), role="vector")
        self.w_in = self.on = None

    def finalize(self, device, dtype) -> None:
        super().finalize(device, dtype)
        self.w_in = self.tensor("in").float().contiguous()
        # what the kernel takes for a pending output: mix [from, to], then out
        self.on = torch.cat([self.tensor("mix").float().reshape(-1), self.tensor("out").float()]).contiguous()


class StreamMix:
    """A sublayer's output ``delta`` that goes into the streams as ``connection`` says."""

    __slots__ = ("delta", "connection")

    def __init__(self, delta, connection: HyperConnection) -> None:
        self.delta = delta
        self.connection = connection
