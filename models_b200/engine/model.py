"""The decoder put together from parts, as its ModelSpec says: embedding, the scheduled runs of
blocks, final norm, output head (integrallis/models' layer order:
backend-java/.../llama/LlamaForwardPass.java:1024-1196).  Every piece, the embedding and the head
included, is built from its spec through the registry of parts; this file knows none of them.
"""

from __future__ import annotations

from typing import Callable, Dict, List, Mapping, Optional

import torch

from ..config.specs import ModelSpec
from ..kernels import ops
from ..parts import RunContext, Runtime, as_delta, build_part
from ..weights.loader import ParamRequest, check_names_and_shapes


def _collect(requests: List[ParamRequest]) -> Dict[str, ParamRequest]:
    out: Dict[str, ParamRequest] = {}
    for r in requests:
        if r.name in out and tuple(out[r.name].shape) != tuple(r.shape):
            raise ValueError(f"tensor {r.name} is asked for with shapes {out[r.name].shape} and {r.shape}")
        out[r.name] = r
    return out


class DecoderModel:
    """Builds every part on `runtime.device`; `load` hands each part its tensors."""

    def __init__(self, spec: ModelSpec, runtime: Runtime):
        self.spec = spec
        self.runtime = runtime
        self.blocks = [build_part("block", layer, runtime) for layer in spec.layers]
        self.final_norm = build_part("norm", spec.final_norm, runtime)
        self.embedding = build_part("embedding", spec.embedding, runtime)
        self.head = build_part("head", spec.head, runtime)
        self.join = build_part("join", spec.join, runtime) if spec.join is not None else None
        # when set, called with (run index, a copy of the float32 residual stream after that run), for
        # finding the layer where two computations part (the reference's LayerObserver,
        # backend-java/.../llama/LlamaForwardPass.java:44-47,1179-1181)
        self.observer: Optional[Callable[[int, torch.Tensor], None]] = None
        self.fused_decode = None  # the whole decode step as one kernel, where the model's parts allow it (set by `load`)

    # ------------------------------------------------------------------ weights

    def parameters(self) -> Dict[str, ParamRequest]:
        requests = list(self.embedding.parameters())
        for block in self.blocks:
            requests += block.parameters()
        requests += self.final_norm.parameters()
        requests += self.head.parameters()
        if self.join is not None:
            requests += self.join.parameters()
        return _collect(requests)

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        requests = self.parameters()
        check_names_and_shapes(requests, {n: tuple(t.shape) for n, t in tensors.items()}, "model tensors")
        self.embedding.load(tensors)
        for block in self.blocks:
            block.load(tensors)
        self.final_norm.load(tensors)
        # tied output: the embedding matrix stands in (backend-java/.../llama/LlamaWeights.java:83-89)
        self.head.load(tensors, tied_to=getattr(self.embedding, "weight", None) if self.spec.head.tied else None)
        if self.join is not None:
            self.join.load(tensors)
        if self.runtime.mode == "bfloat16" and self.runtime.device.type == "cuda":
            from .fused_decode import FusedDecode

            self.fused_decode = FusedDecode(self)

    # ------------------------------------------------------------------ cache needs

    def kv_requests(self):
        return [self.blocks[entry.layer].mixer.kv_request() for entry in self.spec.schedule]

    def state_requests(self):
        return [self.blocks[entry.layer].mixer.state_request() for entry in self.spec.schedule]

    # ------------------------------------------------------------------ forward

    def forward(self, batch, runs: List[RunContext]) -> Optional[torch.Tensor]:
        """Runs the tokens of `batch` through every scheduled run and returns float32 logits at
        batch.want_rows ([rows, vocab]), or None when no row is wanted."""
        if self.fused_decode is not None and self.fused_decode.takes(batch):
            logits = self.fused_decode.run(batch, runs)  # one token for each of a few sequences: the step as one kernel
            if logits is not None:
                return logits
        x = self.embedding.forward(batch.tokens)
        streams = self.spec.residual_streams
        if streams > 1:
            x = ops.stream_copies(x, streams)  # [tokens, streams * width]: every copy starts as the embedding's row
        pending = None
        schedule = self.spec.schedule
        if self.join is not None:
            self.join.begin(x, at_once=schedule[0].joins)
        for index, (run, entry) in enumerate(zip(runs, schedule)):
            block = self.blocks[entry.layer]
            if entry.joins:
                if as_delta(pending) is not None:
                    ops.residual_add(x, as_delta(pending))
                x, pending = self.join.forward(x, pending), None
            after = schedule[index + 1] if index + 1 < len(schedule) else None
            if getattr(block, "takes_next_norm", False):
                # what reads the stream after this run: a join, the next run's first norm, or the final norm
                if after is None:
                    next_norm = self.final_norm
                else:
                    next_norm = self.join if after.joins else getattr(self.blocks[after.layer], "mixer_norm", None)
                pending = block.forward(x, pending, batch, run, next_norm)
            elif getattr(block, "takes_next_block", False):
                # the block that reads the streams after this run (none after the last one): its reading may ride in this one's writing
                following = self.blocks[after.layer] if after is not None and not after.joins else None
                pending = block.forward(x, pending, batch, run, following)
            else:
                pending = block.forward(x, as_delta(pending), batch, run)
            if self.observer is not None:
                delta = as_delta(pending)
                seen = ops.stream_sum(x, self.spec.hidden_size) if streams > 1 else x
                self.observer(run.run, seen + delta.float() if delta is not None else seen.clone())
        if self.join is not None:
            self.join.end()
        if batch.num_wanted == 0:
            return None
        if streams > 1:
            x = ops.stream_sum(x, self.spec.hidden_size)  # the copies added up: what the final norm reads
        if getattr(self.head, "takes_prenormed", False):
            every_row = batch.max_q_len == 1 and batch.num_wanted == batch.num_tokens
            return self.head.forward(x, pending, self.final_norm, batch.want_rows, every_row)
        return self.head.forward(x, as_delta(pending), self.final_norm, batch.want_rows)


def parameter_requests(spec: ModelSpec) -> Dict[str, ParamRequest]:
    """The tensors a model of this spec needs, without building anything on a device."""
    model = DecoderModel(spec, Runtime(torch.device("meta"), "float32", max_positions=1))
    return model.parameters()
