"""A state-space recurrence with one decay per head and token (the scalar form of Mamba-2).

One first product, laid out [z | x | B | C | dt]; x, B and C pass a short causal convolution with a bias and a silu;
dt = softplus(dt + dt_bias); per head (which uses group h / (heads / groups)):

    S <- exp(-exp(A_log) dt) S + dt B x^T;      y = S^T C + D x

then y * silu(z), an RMS norm over equal parts of the row, a gain, and the output matrix.  The per-sequence state is float32 and
lives in the engine's state area: S [heads, state, value_dim], then the convolution's last conv_taps - 1 inputs
[conv_taps - 1, channels].

A decode step, a short step and the 32-bit mode walk the tokens one by one.  A long step in the bfloat16 mode is cut into chunks:
inside one the recurrence is two matrix products with the decays between the chunk's tokens as factors, and only the states at
the chunks' borders follow one another.
"""

from __future__ import annotations

import torch

from ..cache.state import StateRequest
from ..kernels import ops
from ..weights.loader import ParamRequest
from .base import Mixer, RunContext
from .linear import stack_rows
from .registry import register_part
from .split import SplitPart


class StateSpaceMixer(SplitPart, Mixer):
    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        if spec.num_heads % spec.groups:
            raise ValueError(f"{spec.num_heads} heads are no multiple of {spec.groups} groups")
        self.inner_width = spec.num_heads * spec.value_dim
        if self.inner_width % spec.norm_groups:
            raise ValueError(f"{self.inner_width} numbers do not form {spec.norm_groups} equal parts")
        if spec.conv_taps < 1:
            raise ValueError(f"a convolution has at least one weight per channel, got {spec.conv_taps}")
        self.channels = self.inner_width + 2 * spec.groups * spec.state_size
        self.state_floats = spec.num_heads * spec.state_size * spec.value_dim  # S; the convolution's tail follows

    def parameters(self):
        s, n = self.spec, self.spec.weights
        W, H, inner = s.hidden_size, s.num_heads, self.inner_width
        return [ParamRequest(n["in"], (inner + self.channels + H, W)), ParamRequest(n["conv"], (self.channels, s.conv_taps), "bias"),
                ParamRequest(n["conv_bias"], (self.channels,), "bias"), ParamRequest(n["A_log"], (H,), "bias"),
                ParamRequest(n["dt_bias"], (H,), "bias"), ParamRequest(n["D"], (H,), "gain"), ParamRequest(n["norm"], (inner,), "gain"),
                ParamRequest(n["o"], (W, inner))]

    def load(self, tensors):
        n, rt = self.spec.weights, self.runtime
        inner = self.inner_width
        first = rt.matrix(tensors[n["in"]])
        self.w_in, self.starts = stack_rows([first[:inner], first[inner:inner + self.channels], first[inner + self.channels:]])
        self.w_o = rt.matrix(tensors[n["o"]])
        self.conv = rt.vector(tensors[n["conv"]])
        self.conv_bias = rt.vector(tensors[n["conv_bias"]])
        self.decay = (-torch.exp(rt.vector(tensors[n["A_log"]]))).contiguous()
        self.dt_bias = rt.vector(tensors[n["dt_bias"]])
        self.skip = rt.vector(tensors[n["D"]])
        self.gain = rt.vector(tensors[n["norm"]])

    def input_matrix(self):
        return self.w_in

    def output_matrix(self):
        return self.w_o

    def state_request(self):
        floats = self.state_floats + (self.spec.conv_taps - 1) * self.channels
        return StateRequest((-(-floats // 4) * 4,), torch.float32)  # (rows of whole 16-byte pieces)

    def inner(self, proj: torch.Tensor, mid: torch.Tensor, batch, run: RunContext, scale: float = 1.0) -> None:
        s = self.spec
        if run.state is None:
            raise RuntimeError("the state-space recurrence needs its per-sequence state; its run has none")
        at, H, inner = self.starts, s.num_heads, self.inner_width
        z, xbc, dt = proj[:, at[0]:at[0] + inner], proj[:, at[1]:at[1] + self.channels], proj[:, at[2]:at[2] + H]
        b_at = inner
        c_at = inner + s.groups * s.state_size
        chunked = ops.state_space_chunks_takes(proj.dtype, s.state_size, s.value_dim, batch.max_q_len, b_at)
        conv = ops.short_conv(xbc, self.conv, run.state, self.state_floats, batch.slots, batch.cu_q, batch.max_q_len,
                              out_bias=self.conv_bias, activation="silu", store_tail=True,
                              out_dtype=torch.bfloat16 if chunked else torch.float32)
        sizes = (H, s.groups, s.state_size, s.value_dim)
        if chunked:
            y = ops.state_space_chunks(conv, 0, b_at, c_at, dt, self.decay, self.dt_bias, self.skip, run.state, 0, batch.slots, batch.cu_q,
                                       batch.max_q_len, *sizes)
        else:
            y = ops.state_space_walk(conv, 0, b_at, c_at, dt, self.decay, self.dt_bias, self.skip, run.state, 0, batch.slots, batch.cu_q, *sizes)
        ops.gate_part_norm(y, z, self.gain, s.eps, s.norm_groups, mid, scale)


register_part("mixer", "state_space", StateSpaceMixer)
