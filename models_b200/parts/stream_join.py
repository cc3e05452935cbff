"""The residual stream made anew from itself and the embedding's rows: x <- W [x; x_0], ahead of the runs the schedule names (the
passes of a looped span).

The two lie side by side in one row buffer [tokens, 2 * width] in the compute type: `begin` stores x_0 once per step, a join stores
x beside it and runs one product over both.  A block before a join may leave x there itself (`rows_for_stream`), as it makes the rows
a norm will read: with a gain of ones the rows are the stream's own (`weight` and `foldable` are those of such a norm).
"""

from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import ParamRequest
from .base import Part, Prenormed
from .linear import linear
from .registry import register_part


class LinearJoin(Part):
    foldable = True

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.width = spec.hidden_size
        self.matrix = self.rows = self.weight = None
        self.left_stored = False

    def parameters(self):
        return [ParamRequest(self.spec.weights["weight"], (self.width, 2 * self.width))]

    def load(self, tensors):
        self.matrix = self.runtime.matrix(tensors[self.spec.weights["weight"]])
        self.weight = torch.ones((self.width,), dtype=torch.float32, device=self.matrix.device)

    def begin(self, x: torch.Tensor, at_once: bool) -> None:
        """Keeps the embedding's rows x of this step; `at_once`: the first join comes before anything is added to them."""
        self.rows = torch.empty((x.shape[0], 2 * self.width), dtype=self.runtime.compute_dtype, device=x.device)
        ops.store_columns(x, self.rows[:, self.width:], self.rows[:, :self.width] if at_once else None)
        self.left_stored = at_once

    def end(self) -> None:
        self.rows = None

    def rows_for_stream(self) -> torch.Tensor:
        return self.rows[:, :self.width]

    def forward(self, x: torch.Tensor, pending) -> torch.Tensor:
        """The new stream; x is up to date, and already in its place if `pending` is a Prenormed a block made for this join."""
        stored = self.left_stored or (isinstance(pending, Prenormed) and pending.norm is self
                                      and pending.rows.data_ptr() == self.rows.data_ptr())
        if not stored:
            ops.store_columns(x, self.rows[:, :self.width])
        self.left_stored = False
        return linear(self.rows, self.matrix, torch.float32)


register_part("join", "linear_join", LinearJoin)
