"""Dynamic tanh: tanh(alpha * x) * weight + bias, element by element; a norm that computes no mean and no variance.  All of it
in float32 on the float32 residual stream.

Having no row-wise sum, it may stand anywhere: `add_result` puts it between a sublayer's result and the stream (x += norm(y)) and
lets the next reader's norm ride in the same kernel; `then_args` is what such a kernel needs of the norm that reads next.
"""

from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from ..weights.loader import ParamRequest
from .base import Part
from .registry import register_part


class DynamicTanh(Part):
    foldable = False  # no product carries this norm in its prologue

    def parameters(self):
        n = self.spec.weights
        return [ParamRequest(n["weight"], (self.spec.size,), "gain"), ParamRequest(n["bias"], (self.spec.size,), "bias"),
                ParamRequest(n["alpha"], (), "gain")]

    def load(self, tensors):
        n = self.spec.weights
        self.weight = self.runtime.vector(tensors[n["weight"]])
        self.bias = self.runtime.vector(tensors[n["bias"]])
        self.alpha = float(tensors[n["alpha"]].float())

    def forward(self, x: torch.Tensor, delta: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None,
                write_x: bool = True) -> torch.Tensor:
        """x += delta (if any), then the norm of x, or of the rows of x that `rows` picks."""
        if delta is not None:
            ops.residual_add(x, delta)
        return ops.dynamic_tanh(x, self.alpha, self.weight, self.bias, self.runtime.compute_dtype, rows)

    def then_args(self):
        return self.alpha, self.weight, self.bias

    def add_result(self, x: torch.Tensor, y, then) -> Optional[torch.Tensor]:
        """x += norm(y).  y: float32 rows, or an ExpertResults; `then`: see ops.result_tanh_add."""
        entries = {}
        if not isinstance(y, torch.Tensor):
            entries = dict(top=y.top, position=y.position, entry_weight=y.weight)
            y = y.rows
        return ops.result_tanh_add(x, y, self.alpha, self.weight, self.bias, then, self.runtime.compute_dtype, **entries)

    def add_product(self, x: torch.Tensor, a: torch.Tensor, weight: torch.Tensor, then):
        """x += norm(a . weight^T), or None if the product's kernel has no such epilogue (many rows, other types or sizes): with few
        rows (decode) norm, addition and the next reader's rows ride in the product.  Returns (rows of `then`,)."""
        if (self.runtime.mode == "bfloat16" and weight.dtype == torch.bfloat16 and a.dtype == torch.bfloat16 and ops.skinny_pays(weight, a.shape[0])
                and a.stride(0) % 8 == 0 and a.data_ptr() % 16 == 0):
            return (ops.skinny_gemm_tanh_residual(weight, a, x, self.alpha, self.weight, self.bias, then),)
        return None


register_part("norm", "dynamic_tanh", DynamicTanh)
