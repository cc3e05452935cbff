"""Softmax attention whose keys and values are expanded from one low-rank row per position.

q = Wq.xn (heads of `head_dim`); c = rmsnorm(Wd.xn) with a gain, `latent_dim` numbers: the only thing the cache keeps
(one "key head" of latent_dim, no values).  Head h has k_j = Uk_h.c_j and v_j = Uv_h.c_j, so its score
scale * q_i.k_j equals scale * (Uk_h^T q_i).c_j and its result sum_j w_j v_j equals Uv_h.(sum_j w_j c_j): the query is taken
into the latent space once per token and head, the attention runs over the cached rows themselves (all heads read the same
rows, as key and as value), and the result is taken out of the latent space once per token and head.  No key or value of
the cache is ever expanded.  With `gated`, head h's result is multiplied by sigmoid((Wg.xn)_h); then Wo.  The
norm, the scores and the softmax are float32 in both modes.

Variations (the spec says which).  Queries from a latent of their own, q = Uq.rmsnorm(Wdq.xn).  A position: every query head has
`rotary_dim` coordinates more and the cached row as many more, one rotated key part that all heads share; the query in the latent
space is [Uk_h^T q | rotated part], the cached row [c | rotated part], and their product is the whole score; the values are the
row's first latent_dim numbers.  (Rotated pairs (2i, 2i + 1) are brought side by side when the weights are loaded: the rotated
parts meet in dot products only, so the order of their coordinates is nobody's business but theirs, and the kernels know one
pairing.)  A window.  A gate per element.  Rows that another run cached (`own_rows` False).

A prompt that starts its sequences sees no row but its own, and there the other order is cheaper: one product expands every row of
the step into the heads' keys and values, and the attention runs over those (with the shared rotated part beside them), a third of the
multiplications per query and key.  Steps that continue a sequence, and sizes the kernel does not take, stay in the latent space.
"""

from __future__ import annotations

import torch

from ..cache.kv_cache import KvRequest
from ..kernels import ops
from ..weights.loader import ParamRequest
from .base import Mixer, RunContext
from .linear import linear, stack_columns, stack_rows
from .registry import build_part, register_part
from .split import SplitPart


def _whole(size: int) -> int:
    """The next multiple of 64: the columns of a shared-memory tile."""
    return -(-size // 64) * 64


class LatentAttentionMixer(SplitPart, Mixer):
    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        if spec.gate_kind not in ("head", "element"):
            raise ValueError(f"a gate of kind {spec.gate_kind!r} is not built (known: head, element)")
        self.turned = spec.position.rotary_dim if spec.position is not None else 0
        self.q_width = spec.num_heads * (spec.head_dim + self.turned)
        self.row_width = spec.latent_dim + self.turned
        self.mid_width = spec.num_heads * spec.value_dim
        self.rope = None
        if spec.position is not None:
            key = ("position", spec.position, runtime.max_positions)
            if key not in runtime.shared:
                runtime.shared[key] = build_part("position", spec.position, runtime)
            self.rope = runtime.shared[key]

    def _first(self):
        """The matrices that read the normalised rows: (role, rows)."""
        s = self.spec
        out = [("down_q", s.query_latent) if s.query_latent else ("q", self.q_width)]
        if s.own_rows:
            out.append(("down", self.row_width))
        if s.gated:
            out.append(("gate", s.num_heads if s.gate_kind == "head" else self.mid_width))
        return out

    def _paired(self, matrix: torch.Tensor, parts: int) -> torch.Tensor:
        """The rows of `parts` equal parts, each ending in the rotated coordinates, with those ordered as pairs
        (i, i + rotary_dim / 2)."""
        if not self.turned or self.spec.position.pairing == "half":
            return matrix
        size = matrix.shape[0] // parts
        kept = size - self.turned
        order = list(range(kept)) + list(range(kept, size, 2)) + list(range(kept + 1, size, 2))
        return matrix.view(parts, size, -1)[:, torch.tensor(order, device=matrix.device)].reshape(matrix.shape).contiguous()

    def parameters(self):
        s, n = self.spec, self.spec.weights
        out = [ParamRequest(n[role], (rows, s.hidden_size)) for role, rows in self._first()]
        if s.query_latent:
            out += [ParamRequest(n["down_q_norm"], (s.query_latent,), "gain"), ParamRequest(n["up_q"], (self.q_width, s.query_latent))]
        if s.own_rows:
            out.append(ParamRequest(n["down_norm"], (s.latent_dim,), "gain"))
        out += [ParamRequest(n["up_k"], (s.num_heads * s.head_dim, s.latent_dim)),
                ParamRequest(n["up_v"], (self.mid_width, s.latent_dim)),
                ParamRequest(n["o"], (s.hidden_size, self.mid_width))]
        return out

    def load(self, tensors):
        s, n, rt = self.spec, self.spec.weights, self.runtime
        parts = {"q": s.num_heads, "down": 1}  # which of the first matrices end in rotated rows, and how often
        first = [rt.matrix(tensors[n[role]]) for role, _ in self._first()]
        first = [self._paired(m, parts[role]) if role in parts else m for m, (role, _) in zip(first, self._first())]
        if len({m.dtype for m in first}) > 1:
            first = [m.float() for m in first]
        self.w_in, starts = stack_rows(first)
        self.columns = {role: slice(at, at + rows) for (role, rows), at in zip(self._first(), starts)}
        self.w_o = rt.matrix(tensors[n["o"]])
        self.latent_gain = rt.vector(tensors[n["down_norm"]]) if s.own_rows else None
        if s.query_latent:
            self.query_gain = rt.vector(tensors[n["down_q_norm"]])
            self.up_q, _, _ = stack_columns([self._paired(rt.matrix(tensors[n["up_q"]]), s.num_heads)])  # (columns of padding meet zeros)
        dtype = rt.compute_dtype
        # per head: [latent_dim, head_dim] takes a query into the latent space, [value_dim, latent_dim] a result out of it
        self.into_latent = rt.matrix(tensors[n["up_k"]]).to(dtype).view(s.num_heads, s.head_dim, s.latent_dim).transpose(1, 2).contiguous()
        self.out_of_latent = rt.matrix(tensors[n["up_v"]]).to(dtype).view(s.num_heads, s.value_dim, s.latent_dim).contiguous()

        self.expand = None
        K, D, V = s.latent_dim, s.head_dim, s.value_dim
        if (rt.mode == "bfloat16" and s.own_rows and not s.query_latent and (not s.gated or s.gate_kind == "head") and K % 8 == 0
                and (D + self.turned) % 8 == 0 and V % 8 == 0 and V <= 128 and _whole(D) + _whole(self.turned) <= 256):
            # every head's key and value matrices padded with zero rows to whole 64s: [heads * keys; heads * values] x latent
            pad = lambda m, size: torch.nn.functional.pad(m, (0, 0, 0, _whole(size) - size)).reshape(-1, K)  # noqa: E731
            self.expand = torch.cat([pad(rt.matrix(tensors[n["up_k"]]).to(dtype).view(s.num_heads, D, K), D),
                                     pad(self.out_of_latent, V)]).contiguous()

    @property
    def starts_differ(self) -> bool:
        """Whether prompts that start their sequences take another way than steps that continue them."""
        return getattr(self, "expand", None) is not None

    def input_matrix(self):
        return self.w_in

    def output_matrix(self):
        return self.w_o

    def kv_request(self):
        # one row per position, read as key and as value
        return KvRequest(1, self.row_width, self.spec.window, 0)

    def inner(self, proj: torch.Tensor, mid: torch.Tensor, batch, run: RunContext, scale: float = 1.0) -> None:
        s = self.spec
        if run.k_pool is None:
            raise RuntimeError("the latent attention mixer needs a cache pool; its run has none")
        if run.writes_cache != s.own_rows:
            raise RuntimeError("this mixer makes rows of its own and its run reads another's, or the other way round")
        if scale != 1.0:
            raise ValueError("this mixer's result cannot be scaled on its way out")
        group = batch.groups[run.group]
        part = lambda role: proj[:, self.columns[role]] if role in self.columns else None  # noqa: E731
        cos, sin = (self.rope.cos, self.rope.sin) if self.rope is not None else (None, None)
        down_q, down, gate = part("down_q"), part("down"), part("gate")
        q_rows = None
        if down_q is None and down is not None:
            q = part("q")
            fresh = (self.expand is not None and getattr(batch, "fresh", False) and batch.max_q_len >= ops.TCGEN05_ATTENTION_MIN_ROWS
                     and q.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0 and mid.stride(0) % 8 == 0 and mid.data_ptr() % 16 == 0)
            more = {"q": q, "heads": s.num_heads, "head_columns": s.head_dim + self.turned, "padded": _whole(self.turned)} if fresh else {}
            own, tail, q_tail = ops.latent_rows(down, self.latent_gain, self.turned, cos, sin, batch.positions, s.eps, run.k_pool,
                                                group.slot_mapping, **more)
            if fresh:
                at = s.num_heads * _whole(s.head_dim)
                expanded = linear(own, self.expand, own.dtype)
                ops.prompt_attention(q, q_tail, expanded[:, :at], expanded[:, at:], tail, mid, batch.cu_q, batch.kv_lens, batch.max_q_len,
                                     s.num_heads, s.head_dim + self.turned, s.value_dim, s.scale, gate, s.window or 0)
                return
        elif down_q is not None:
            q_rows = ops.latent_prepare(down_q, self.query_gain if down_q is not None else None, self.up_q.shape[1] if down_q is not None else 0,
                                        down, self.latent_gain, self.turned, cos, sin, batch.positions, s.eps, run.k_pool, group.slot_mapping)
        q = part("q") if down_q is None else linear(q_rows, self.up_q, proj.dtype)
        rows = proj.shape[0]
        q_latent = torch.empty((rows, s.num_heads * self.row_width), dtype=proj.dtype, device=proj.device)
        ops.head_linear(q, self.into_latent, q_latent, s.num_heads, turned=self.turned, cos=cos, sin=sin, positions=batch.positions)
        mixed = torch.empty((rows, s.num_heads * s.latent_dim), dtype=proj.dtype, device=proj.device)
        ops.gated_attention(q_latent, mixed, run.k_pool, None, group.block_table, batch.cu_q, batch.kv_lens, batch.max_q_len,
                            s.num_heads, 1, self.row_width, s.latent_dim, "softmax", s.scale, window=s.window or 0)
        ops.head_linear(mixed, self.out_of_latent, mid, s.num_heads, gate, gate_kind=s.gate_kind)


register_part("mixer", "latent_attention", LatentAttentionMixer)
