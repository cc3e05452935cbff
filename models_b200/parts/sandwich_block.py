"""A layer with a norm before and after each sublayer, and (where the spec asks for it) the token let in once more at its end:

    x += mixer_out_norm(mixer(mixer_norm(x)))
    x += feed_forward_out_norm(feed_forward(feed_forward_norm(x)))      (if the layer has a feed-forward)
    x += side_norm(side(x))                                             (if it has a side input)

The norms before a sublayer are dynamic tanhs: they need no sum over a row, so the kernel that adds a sublayer's result into the
float32 stream also makes the next reader's rows -- the feed-forward's, the side input's (the stream itself in the compute type),
and, handed on as StreamRows, the next layer's.  The norms on the results offer `add_result` (a dynamic tanh, an RMS norm).
A sublayer is a part with `forward_results` (expert results still to be summed), with `forward_wide` (float32 rows), or a split
part (a first product, something in between, a last product whose float32 sums are the result; with few rows the norm on
the result and the addition ride in that product's epilogue where the norm offers it, `add_product`).
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import Part, RunContext, StreamRows, as_delta
from .linear import linear
from .registry import build_part, register_part


class SandwichBlock(Part):
    takes_next_block = True  # `forward` is told which block runs next

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        build = lambda sort, s: build_part(sort, s, runtime) if s is not None else None  # noqa: E731
        self.mixer_norm, self.mixer, self.mixer_out_norm = build("norm", spec.mixer_norm), build("mixer", spec.mixer), build("norm", spec.mixer_out_norm)
        self.feed_forward_norm, self.feed_forward = build("norm", spec.feed_forward_norm), build("feed_forward", spec.feed_forward)
        self.feed_forward_out_norm = build("norm", spec.feed_forward_out_norm)
        self.side, self.side_norm = build("feed_forward", spec.side), build("norm", spec.side_norm)
        self.sublayers = [(self.mixer_norm, self.mixer, self.mixer_out_norm)]  # (norm before or None, part, norm on the result)
        if self.feed_forward is not None:
            self.sublayers.append((self.feed_forward_norm, self.feed_forward, self.feed_forward_out_norm))
        if self.side is not None:
            self.sublayers.append((None, self.side, self.side_norm))
        for before, part, after in self.sublayers:
            if before is not None and not hasattr(before, "then_args"):
                raise ValueError(f"{type(before).__name__} cannot ride in the addition before it: this block cannot run it before a sublayer")
            if not hasattr(after, "add_result"):
                raise ValueError(f"{type(after).__name__} has no add_result: this block cannot run it on a result")
            if not any(hasattr(part, name) for name in ("forward_results", "forward_wide")) \
                    and not all(hasattr(part, name) for name in ("input_matrix", "output_matrix", "inner")):
                raise ValueError(f"{type(part).__name__} is neither a split part nor one with float32 results: this block cannot run it")
        self.parts = [p for sublayer in self.sublayers for p in sublayer if p is not None]

    def parameters(self):
        return [p for part in self.parts for p in part.parameters()]

    def load(self, tensors):
        for part in self.parts:
            part.load(tensors)

    def _sublayer(self, x, part, after, rows, batch, run, then):
        """x += after(part(rows)); returns the rows that `then` asks for."""
        if hasattr(part, "forward_results"):
            return after.add_result(x, part.forward_results(rows, batch, run), then)
        if hasattr(part, "forward_wide"):
            return after.add_result(x, part.forward_wide(rows, batch, run), then)
        dtype = self.runtime.compute_dtype
        w_in, w_out = part.input_matrix(), part.output_matrix()
        proj = linear(rows, w_in, dtype)
        mid = torch.empty((rows.shape[0], w_out.shape[1]), dtype=dtype, device=rows.device)
        part.inner(proj[:, :w_in.shape[0]], mid, batch, run, 1.0)
        done = after.add_product(x, mid, w_out, then) if hasattr(after, "add_product") else None
        return done[0] if done is not None else after.add_result(x, linear(mid, w_out, torch.float32), then)

    def forward(self, x: torch.Tensor, pending, batch, run: RunContext, following=None):
        """`pending`: None, a delta still to be added, or the rows the block before left for this one (a StreamRows).
        `following`: the block that runs next; if it is one of these, it is handed its first norm's rows."""
        rows = None
        if isinstance(pending, StreamRows):
            rows = pending.rows if pending.reader is self else None
        elif as_delta(pending) is not None:
            ops.residual_add(x, as_delta(pending))
        if rows is None:
            rows = self.mixer_norm.forward(x)
        hand_on = isinstance(following, SandwichBlock)
        float_mode = self.runtime.compute_dtype == torch.float32
        for i, (_, part, after) in enumerate(self.sublayers):
            if i + 1 < len(self.sublayers):
                before = self.sublayers[i + 1][0]
                # (in the 32-bit mode a reader of the stream itself reads x: nothing is copied)
                then = before.then_args() if before is not None else (None if float_mode else "rows")
            else:
                then = following.mixer_norm.then_args() if hand_on else None
            rows = self._sublayer(x, part, after, rows, batch, run, then)
            if rows is None:
                rows = x
        return StreamRows(rows, following) if hand_on else None


register_part("block", "sandwich", SandwichBlock)
