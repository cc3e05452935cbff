"""Dense gated feed-forward with clamped branches: down(g * sigmoid(slope * g) * (u + up_offset)) with g = min(gate(xn), limit) and
u = clamp(up(xn), -limit, limit).

A split part (parts/split.py) whose first matrix is [gate rows; up rows], so a block can run both branches and what becomes of
them as ONE product (`pair_epilogue`: the constants of the product's epilogue); `inner` is the same as a kernel of its own.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import ParamRequest
from .base import Part
from .linear import stack_rows
from .registry import register_part
from .split import SplitPart


class ClampedFeedForward(SplitPart, Part):
    def parameters(self):
        s, n = self.spec, self.spec.weights
        size = s.expert.intermediate_size
        return [ParamRequest(n["gate"], (size, s.hidden_size)), ParamRequest(n["up"], (size, s.hidden_size)),
                ParamRequest(n["down"], (s.hidden_size, size))]

    def load(self, tensors):
        n, rt = self.spec.weights, self.runtime
        first = [rt.matrix(tensors[n[r]]) for r in ("gate", "up")]
        if first[0].dtype != first[1].dtype:
            first = [m.float() for m in first]
        self.w_in, (_, self.up_at) = stack_rows(first)
        self.w_down = rt.matrix(tensors[n["down"]])

    def input_matrix(self):
        return self.w_in

    def output_matrix(self):
        return self.w_down

    def pair_epilogue(self):
        """(limit, slope, up_offset) for a product over [gate rows; up rows] that stores the gated results, or None where padding
        lies between the two."""
        e = self.spec.expert
        return (e.limit, e.swish_slope, e.up_offset) if self.up_at == e.intermediate_size else None

    def inner(self, proj: torch.Tensor, mid: torch.Tensor, batch=None, run=None, scale: float = 1.0) -> None:
        if scale != 1.0:
            raise ValueError("this feed-forward's result cannot be scaled on its way out")
        e, size = self.spec.expert, self.spec.expert.intermediate_size
        ops.clamped_swish(proj[:, :size], proj[:, self.up_at:self.up_at + size], mid[:, :size], e.limit, e.swish_slope, e.up_offset)

    def forward(self, xn: torch.Tensor, batch=None, run=None) -> torch.Tensor:
        return SplitPart.forward(self, xn)


register_part("feed_forward", "clamped", ClampedFeedForward)
