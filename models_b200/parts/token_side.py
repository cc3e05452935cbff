"""The token itself, let in once more beside the stream: y = P . (gelu_tanh(G . x) * e), with e this layer's columns of the
token's row of a second table.  A layer keeps its own columns of the table, so that a token's numbers lie together.  The
gates' arithmetic is float32; `forward_wide` returns the float32 sums of the last product.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import ParamRequest
from .base import Part
from .linear import linear, stack_columns, stack_rows
from .registry import register_part


class TokenSide(Part):
    def parameters(self):
        s, n = self.spec, self.spec.weights
        return [ParamRequest(n["table"], (s.vocab_size, s.layers * s.dim)), ParamRequest(n["gate"], (s.dim, s.hidden_size)),
                ParamRequest(n["proj"], (s.hidden_size, s.dim))]

    def load(self, tensors):
        s, n, rt = self.spec, self.spec.weights, self.runtime
        self.table = rt.matrix(tensors[n["table"]][:, s.index * s.dim:(s.index + 1) * s.dim])
        # (rows and columns of padding up to a multiple of 8, so that the package's own products take any size)
        self.gate, _ = stack_rows([rt.matrix(tensors[n["gate"]])])
        self.proj, _, _ = stack_columns([rt.matrix(tensors[n["proj"]])])
        self.table = self.table.to(rt.compute_dtype)

    def forward_wide(self, xn: torch.Tensor, batch, run=None) -> torch.Tensor:
        """xn: the stream's rows in the compute type; float32 [tokens, width]."""
        if (xn.dtype == torch.bfloat16 and self.gate.dtype == torch.bfloat16 and ops.skinny_pays(self.gate, xn.shape[0])
                and xn.stride(0) % 8 == 0 and xn.data_ptr() % 16 == 0):
            gated = ops.skinny_gemm_side(self.gate, xn, self.table, batch.tokens, self.proj.shape[1])  # few rows: in the product's epilogue
        else:
            gated = ops.side_gate(linear(xn, self.gate, torch.float32), self.table, batch.tokens, self.proj.shape[1])
        return linear(gated, self.proj, torch.float32)


register_part("feed_forward", "token_side", TokenSide)
