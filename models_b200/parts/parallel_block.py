"""A layer with ONE norm whose rows feed the mixer and the feed-forward side by side:
h = norm(x); x += mixer(h) + feed_forward(h).

Both sublayers are split parts (parts/split.py), so the layer is two matrix products with the parts' own
kernels between them: every first matrix of the layer, stacked, times h; then each part turns its columns
of that result into its columns of the last product's input; then the last matrices, side by side, times
that input, added into the float32 residual stream in the product's epilogue.  The sum over the sublayers
is thus part of the product's float32 accumulation.

Where the norm's gain can be folded, it rides in the products around it for up to 128 rows: the last product leaves the next
reader's rows (handed on as a Prenormed), the first one divides by the root mean square in its epilogue; with few rows the first
product of a chain normalises the float32 rows itself.  A feed-forward of gate/up pairs (`pair_epilogue`) needs no kernel of its own:
its pairs meet in the first product's epilogue, which stores them as the last product's input -- one product with two kinds
of rows for few activations, two products for more.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import Part, Prenormed, RunContext, as_delta
from .linear import add_linear, linear, stack_columns, stack_rows
from .registry import build_part, register_part


class ParallelBlock(Part):
    takes_next_norm = True  # `forward` is told what reads the stream next, and may hand it a Prenormed

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.norm = build_part("norm", spec.norm, runtime)
        self.mixer_norm = self.norm  # the norm that reads the stream when this layer begins
        self.mixer = build_part("mixer", spec.mixer, runtime)
        self.feed_forward = build_part("feed_forward", spec.feed_forward, runtime) if spec.feed_forward is not None else None
        self.parts = [self.norm, self.mixer] + ([self.feed_forward] if self.feed_forward is not None else [])
        for part in self.parts[1:]:
            if not all(hasattr(part, name) for name in ("input_matrix", "output_matrix", "inner")):
                raise ValueError(f"{type(part).__name__} is no split part: a parallel block cannot run it")

    def parameters(self):
        return [p for part in self.parts for p in part.parameters()]

    def load(self, tensors):
        for part in self.parts:
            part.load(tensors)
        sublayers = self.parts[1:]
        first = [part.input_matrix() for part in sublayers]
        last = [part.output_matrix() for part in sublayers]
        if len({m.dtype for m in first + last}) > 1:
            first, last = [m.float() for m in first], [m.float() for m in last]
        self.w_in, self.in_starts = stack_rows(first)
        self.w_out, self.mid_starts, self.mid_padded = stack_columns(last)
        self.in_widths = [m.shape[0] for m in first]
        self.mid_widths = [m.shape[1] for m in last]
        # the constants of the feed-forward's pairs, where the first product's epilogue can make them
        pairs = getattr(self.feed_forward, "pair_epilogue", None)
        self.pairs = pairs() if pairs is not None and self.runtime.mode == "bfloat16" and self.w_in.dtype == torch.bfloat16 else None
        if self.pairs is not None:
            at = self.in_starts[1]
            self.w_mixer, self.w_pairs = self.w_in[:at], self.w_in[at:at + self.in_widths[1]]

    def _first_product(self, x, pending, mid):
        """(the stacked results of the parts that still need their `inner`, how many parts those are)."""
        rows, norm = x.shape[0], self.norm
        low = self.runtime.mode == "bfloat16"
        ready = pending if isinstance(pending, Prenormed) and pending.norm is norm else None
        some = 1 if self.pairs is not None else len(self.parts) - 1
        pair_columns = mid[:, self.mid_starts[1]:self.mid_starts[1] + self.mid_widths[1]] if self.pairs is not None else None
        if low and getattr(norm, "foldable", False) and ops.skinny_pays(self.w_in, rows, with_norm=True):
            source = {"x": ready.rows, "norm_parts": ready.norm_parts()} if ready is not None \
                else {"xf": x, "gain": norm.weight, "eps": norm.spec.eps}
            if self.pairs is not None:
                return ops.skinny_gemm_pairs(self.w_in, self.in_starts[1], pair_columns, self.pairs, **source), some
            return ops.skinny_gemm(self.w_in, ops.EPI_BF16, **source), some
        on_tiles = low and ops.gemm_tcgen05_takes(self.w_in, rows=rows)
        h, parts = norm.forward(x) if ready is None or not on_tiles else ready.rows, None
        if ready is not None and on_tiles:
            parts = ready.norm_parts()
        if on_tiles and self.pairs is not None and ops.gemm_tcgen05_takes(self.w_pairs, ops.EPI_SWIGLU, rows):
            ops.tensor_core_gemm(h, self.w_pairs, ops.EPI_CLAMPED, out=pair_columns, norm_parts=parts, clamp=self.pairs)
            return ops.tensor_core_gemm(h, self.w_mixer, norm_parts=parts), some
        if on_tiles:
            return ops.tensor_core_gemm(h, self.w_in, norm_parts=parts), len(self.parts) - 1
        return linear(h, self.w_in, self.runtime.compute_dtype), len(self.parts) - 1

    def _last_product(self, x, mid, next_norm):
        """x += mid . w_out^T; a Prenormed where the product left the next reader's rows."""
        rows, w = x.shape[0], self.w_out
        emits = (self.runtime.mode == "bfloat16" and w.dtype == torch.bfloat16 and getattr(next_norm, "foldable", False)
                 and w.shape[0] % 8 == 0)
        few = ops.skinny_pays(w, rows)
        place = getattr(next_norm, "rows_for_stream", None)  # a join takes the stream itself, at a place of its own
        # (a single row gains nothing from a norm's prepared rows: normalising it inside a product costs less than the parts)
        if not emits or not (few and (rows >= 2 or place is not None) or (not few and rows <= ops.WIDE_ROWS and ops.gemm_tcgen05_takes(w, ops.EPI_RESIDUAL, rows))):
            add_linear(x, mid, w)
            return None
        product = ops.skinny_gemm if few else (lambda w, epilogue, x, **more: ops.wide_gemm(x, w, epilogue, **more))
        _, gained, ssq, count = product(w, ops.EPI_RESIDUAL, x=mid, out=x, emit_gain=next_norm.weight,
                                        emit_rows=place() if place is not None else None)
        return Prenormed(gained, ssq, count, x.shape[1], next_norm.spec.eps if place is None else 0.0, next_norm)

    def forward(self, x: torch.Tensor, pending, batch, run: RunContext, next_norm=None):
        if as_delta(pending) is not None:
            ops.residual_add(x, as_delta(pending))
        make = torch.zeros if self.mid_padded else torch.empty
        mid = make((x.shape[0], self.w_out.shape[1]), dtype=self.runtime.compute_dtype, device=x.device)
        proj, count = self._first_product(x, pending, mid)
        for part, a, n, c, m in list(zip(self.parts[1:], self.in_starts, self.in_widths, self.mid_starts, self.mid_widths))[:count]:
            part.inner(proj[:, a:a + n], mid[:, c:c + m], batch, run, 1.0)
        return self._last_product(x, mid, next_norm)


register_part("block", "parallel", ParallelBlock)
