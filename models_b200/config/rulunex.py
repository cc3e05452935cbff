"""Typed configuration of the Rulunex decoder, read from the keys of its own config.json.

A Rulunex layer has ONE norm whose rows both sublayers read: h = N(x); x += mixer(h) + ff(h) (or the mixer alone), with
N(x) = x / rms(x) * (1 + w), the weight stored as its distance from one.  A span of layers runs several times in a row with the same
weights, each pass with a cache of its own; ahead of every pass the stream is made anew from itself and the embedding's rows,
x <- J [x; x_0].  Every layer names its mixer and carries its own sizes and constants:

  "latent_attention"  softmax attention over one cached row per position: an RMS-normed latent that every head expands into its
                      keys and values, and one rotated key part that all heads share; rotary pairs (2i, 2i + 1); a sigmoid gate per
                      head; every earlier position is visible.
  "attention"         grouped-query softmax attention with a sliding window.  The values are the keys as projected; queries and keys
                      pass one RMS norm each over the whole projection before the heads are split; rotary pairs (i, i + dims/2) on
                      the first part of a head, with long wavelengths stretched ("scaling").

The feed-forward is down(g * sigmoid(1.702 g) * (u + 1)) with g = min(gate(h), limit) and u = clamp(up(h), -limit, limit).  The
embedding's rows are multiplied by a scale; the logits are the embedding table itself times N(x).

config.json (every size and constant of a model is here or is a tensor's shape):

    {"architecture": "Rulunex", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads": H, "dim": D, "rot_dim": R, "vdim": Dv, "kv_rank": C, "scale": s, "rot": {"dims": R, "base": b}},
                 "mlp": {"kind": "dense", "ff": F, "limit": l} | null},
                {"type": "attention",
                 "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": s, "mask": {"size": n},
                           "rot": {"dims": r, "base": b, "scaling": {"factor": f, "low": x, "high": y, "original": n}}},
                 "mlp": ...}, ...]}

Tensors: `embed`, `loop.in` (with a loop), `final.norm`, and per layer i under `l<i>.`: `norm1`; `mix.{q,dkv,dkv.norm,uk,uv,g,o}`
(latent_attention), `mix.{q,k,q.norm,k.norm,o}` (attention); `mlp.{gate,up,down}`.  Linear weights are [out, in].
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .kabanex import UNLIMITED_POSITIONS, _float, _get, _int
from .llama import ConfigError
from .specs import (
    ChunkedAttentionSpec,
    ClampedExpertSpec,
    ClampedFeedForwardSpec,
    EmbeddingSpec,
    HeadSpec,
    LatentAttentionSpec,
    ModelSpec,
    NormSpec,
    ParallelBlockSpec,
    RopeScalingSpec,
    RopeSpec,
    ScheduleEntry,
    StreamJoinSpec,
)

ARCHITECTURE = "Rulunex"
MIXERS = ("latent_attention", "attention")
# Constants the design fixes.
SWISH_SLOPE = 1.702  # the gate branch is g * sigmoid(1.702 g)
UP_OFFSET = 1.0      # the up branch is u + 1
GAIN_OFFSET = 1.0    # a layer norm's gain is 1 + w


@dataclass(frozen=True)
class RulunexScaling:
    factor: float
    low: float
    high: float
    original: float  # positions the unstretched frequencies were made for


@dataclass(frozen=True)
class RulunexAttention:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: int     # 0: no "mask", every earlier key is visible
    rot_dims: int   # 0: no rotation
    rot_base: float
    scaling: Optional[RulunexScaling]


@dataclass(frozen=True)
class RulunexLatent:
    heads: int
    dim: int
    rot_dim: int    # 0: no rotated part
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float


@dataclass(frozen=True)
class RulunexFeedForward:
    ff: int
    limit: float


@dataclass(frozen=True)
class RulunexLayer:
    type: str
    mixer: object
    mlp: Optional[RulunexFeedForward]


def _attention(mixer, where: str) -> RulunexAttention:
    heads, kv_heads = _int(mixer, "heads", where), _int(mixer, "kv_heads", where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}.heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    dim = _int(mixer, "dim", where)
    if mixer.get("vdim") is not None and _int(mixer, "vdim", where) != dim:
        raise ConfigError(f"config.json: {where}.vdim ({mixer['vdim']}) must equal dim ({dim}): the values are the projected keys")
    window = _int(mixer["mask"], "size", where + ".mask") if mixer.get("mask") is not None else 0
    dims, base, scaling = 0, 0.0, None
    rot, rw = mixer.get("rot"), where + ".rot"
    if rot is not None:
        dims = _int(rot, "dims", rw, least=0)
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {rw}.dims must be even and at most dim ({dim}), got {dims}")
        base = _float(rot, "base", rw, positive=True)
        if rot.get("scaling") is not None:
            s, sw = rot["scaling"], rw + ".scaling"
            scaling = RulunexScaling(*(_float(s, key, sw, positive=True) for key in ("factor", "low", "high", "original")))
            if scaling.low >= scaling.high:
                raise ConfigError(f"config.json: {sw}.low ({scaling.low}) must lie below high ({scaling.high})")
    return RulunexAttention(heads, kv_heads, dim, _float(mixer, "scale", where), window, dims, base, scaling)


def _latent(mixer, where: str) -> RulunexLatent:
    rot_dim, base = _int(mixer, "rot_dim", where, least=0), 0.0
    if rot_dim:
        rot, rw = _get(mixer, "rot", where), where + ".rot"
        if _int(rot, "dims", rw) != rot_dim or rot_dim % 2:
            raise ConfigError(f"config.json: {rw}.dims must be even and equal to rot_dim ({rot_dim}), got {rot['dims']}")
        base = _float(rot, "base", rw, positive=True)
    return RulunexLatent(_int(mixer, "heads", where), _int(mixer, "dim", where), rot_dim, _int(mixer, "vdim", where),
                         _int(mixer, "kv_rank", where), _float(mixer, "scale", where), base)


def _feed_forward(mlp, where: str) -> Optional[RulunexFeedForward]:
    if mlp is None:
        return None
    if _get(mlp, "kind", where) != "dense":
        raise ConfigError(f"config.json: {where}.kind {mlp['kind']!r} is not built (known: dense)")
    return RulunexFeedForward(_int(mlp, "ff", where), _float(mlp, "limit", where, positive=True))


@dataclass(frozen=True)
class RulunexConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    loop: Optional[Tuple[int, int, int]]  # (start, stop, times)
    layers: Tuple[RulunexLayer, ...]

    @staticmethod
    def from_dict(raw: Mapping[str, Any]) -> "RulunexConfig":
        vocab = _int(raw, "vocab", "the model")
        width = _int(raw, "width", "the model")
        eps = _float(_get(raw, "norm", "the model"), "eps", "norm", positive=True)
        scale = _float(raw["embedding"], "scale", "embedding") if raw.get("embedding") is not None else 1.0
        listed = _get(raw, "layers", "the model")
        if not isinstance(listed, (list, tuple)) or not listed:
            raise ConfigError("config.json: layers must be a non-empty list")
        layers = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]"
            kind = _get(entry, "type", where)
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not built (known: {', '.join(MIXERS)})")
            parse = _attention if kind == "attention" else _latent
            layers.append(RulunexLayer(kind, parse(_get(entry, "mixer", where), where + ".mixer"), _feed_forward(entry.get("mlp"), where + ".mlp")))
        loop = None
        if raw.get("loop") is not None:
            lp = raw["loop"]
            start, stop, times = _int(lp, "start", "loop", least=0), _int(lp, "stop", "loop"), _int(lp, "times", "loop")
            if not start < stop <= len(layers):
                raise ConfigError(f"config.json: loop must satisfy start < stop <= {len(layers)} layers, got {start}, {stop}")
            loop = (start, stop, times)
        return RulunexConfig(str(raw.get("architecture", ARCHITECTURE)), vocab, width, eps, scale, loop, tuple(layers))

    def to_dict(self) -> dict:
        layers = []
        for layer in self.layers:
            m = layer.mixer
            if layer.type == "attention":
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.dim, "scale": m.scale}
                if m.window:
                    mixer["mask"] = {"size": m.window}
                if m.rot_base:
                    mixer["rot"] = {"dims": m.rot_dims, "base": m.rot_base}
                    if m.scaling is not None:
                        s = m.scaling
                        mixer["rot"]["scaling"] = {"factor": s.factor, "low": s.low, "high": s.high, "original": s.original}
            else:
                mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "scale": m.scale}
                if m.rot_dim:
                    mixer["rot"] = {"dims": m.rot_dim, "base": m.rot_base}
            mlp = None if layer.mlp is None else {"kind": "dense", "ff": layer.mlp.ff, "limit": layer.mlp.limit}
            layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "embedding": {"scale": self.embedding_scale}, "layers": layers}
        if self.loop is not None:
            out["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return out

    def schedule(self) -> Tuple[ScheduleEntry, ...]:
        """The runs: the looped span `times` times in a row, the stream joined with the embedding's rows ahead of each pass."""
        n = len(self.layers)
        if self.loop is None:
            return tuple(ScheduleEntry(i) for i in range(n))
        start, stop, times = self.loop
        one_pass = [ScheduleEntry(i, joins=i == start) for i in range(start, stop)]
        return tuple([ScheduleEntry(i) for i in range(start)] + one_pass * times + [ScheduleEntry(i) for i in range(stop, n)])

    def _mixer_spec(self, layer: RulunexLayer, mp: str):
        m, W, eps = layer.mixer, self.width, self.norm_eps
        if layer.type == "latent_attention":
            names = {"q": mp + "q", "down": mp + "dkv", "down_norm": mp + "dkv.norm", "up_k": mp + "uk", "up_v": mp + "uv",
                     "gate": mp + "g", "o": mp + "o"}
            position = RopeSpec(m.rot_dim, m.rot_base, "interleaved") if m.rot_dim else None
            return LatentAttentionSpec(hidden_size=W, num_heads=m.heads, head_dim=m.dim, value_dim=m.vdim, latent_dim=m.kv_rank,
                                       scale=m.scale, eps=eps, gated=True, weights=names, position=position)
        position = None
        if m.rot_dims:
            s = m.scaling
            scaling = None if s is None else RopeScalingSpec("llama3", s.factor, low_freq_factor=s.low, high_freq_factor=s.high,
                                                             original_max_position=s.original)
            position = RopeSpec(m.rot_dims, m.rot_base, "half", scaling)
        names = {"q": mp + "q", "k": mp + "k", "q_norm": mp + "q.norm", "k_norm": mp + "k.norm", "o": mp + "o"}
        return ChunkedAttentionSpec(hidden_size=W, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.dim,
                                    scale=m.scale, eps=eps, position=position, chunk=None, bias=False, projection_norm=True,
                                    weights=names, window=m.window or None, values_from_keys=True)

    def model_spec(self) -> ModelSpec:
        W, eps = self.width, self.norm_eps
        norm = lambda name: NormSpec(W, eps, {"weight": name}, gain_offset=GAIN_OFFSET)  # noqa: E731
        blocks = []
        for i, layer in enumerate(self.layers):
            p, f = f"l{i}.", layer.mlp
            feed_forward = None
            if f is not None:
                feed_forward = ClampedFeedForwardSpec(W, ClampedExpertSpec(f.ff, f.limit, SWISH_SLOPE, UP_OFFSET),
                                                      {r: p + "mlp." + r for r in ("gate", "up", "down")})
            blocks.append(ParallelBlockSpec(mixer=self._mixer_spec(layer, p + "mix."), feed_forward=feed_forward, norm=norm(p + "norm1")))
        return ModelSpec(
            architecture=self.architecture,
            vocab_size=self.vocab,
            hidden_size=W,
            max_positions=UNLIMITED_POSITIONS,
            embedding=EmbeddingSpec(self.vocab, W, self.embedding_scale, {"weight": "embed"}),
            layers=tuple(blocks),
            schedule=self.schedule(),
            final_norm=norm("final.norm"),
            head=HeadSpec(self.vocab, W, True, {}),
            join=StreamJoinSpec(W, {"weight": "loop.in"}) if self.loop is not None else None,
        )
