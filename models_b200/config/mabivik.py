"""Typed configuration of the Mabivik decoder, read from the keys of its own config.json.

A Mabivik layer norms before and after each sublayer with a dynamic tanh, N(x) = tanh(alpha x) * w + b (no mean, no variance):
x += N1b(mixer(N1(x))), then x += N2b(ff(N2(x))) where the layer has a feed-forward, and then lets the token in once more:
x += rms(P (gelu_tanh(G x) * e)), e being the layer's columns of the token's row of a second table.  Every layer names its mixer
and carries its own sizes and constants:

  "delta"             the gated delta rule over q, k, v that pass a short causal convolution and a silu, unit-length q and k, a write
                      strength and a decay per head and token, a float32 state per head, an RMS norm per head and a silu gate.
  "latent_attention"  softmax attention over one cached row per position: an RMS-normed latent that every head expands into its
                      keys and values, and one rotated key part that all heads share.  Queries come from a latent of their own;
                      rotary pairs (i, i + dims/2) with YaRN-stretched frequencies; a sliding window; a gate per element.  A layer
                      with `kv_from` reads the rows of an earlier layer instead of making some.
  "mamba2"            a state-space recurrence with one decay per head and token, behind a short causal convolution; the gate comes
                      before an RMS norm over equal parts of the row.

The feed-forward is a mixture of experts down(silu(gate(h)) * up(h)) without a router: a table of token ids names every token's
experts, each with the weight 1 / top.  The logits are head . N(x), times logit_scale.

config.json (every size and constant of a model is here or is a tensor's shape):

    {"architecture": "Mabivik", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s}, "logit_scale": c,
     "token_side": {"dim": d},
     "layers": [{"type": "delta", "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": Dv, "conv": taps}, "mlp": ...},
                {"type": "latent_attention",
                 "mixer": {"heads": H, "dim": D, "rot_dim": R, "vdim": Dv, "q_rank": Q, "kv_rank": K, "scale": s, "mask": {"size": n},
                           "rot": {"dims": R, "base": b, "scaling": {"factor": f, "original": n, "fast": a, "slow": z}},
                           "kv_from": j (optional)}, "mlp": ...},
                {"type": "mamba2", "mixer": {"heads": H, "vdim": P, "state": N, "groups": G, "norm_groups": M, "conv": taps},
                 "mlp": {"kind": "moe", "router": {"experts": E, "top": k}, "expert": {"ff": F}} | null}, ...]}

Tensors: `embed`, `side.embed`, `head`, `final.norm`, and per layer i under `l<i>.`: `norm1`, `norm1b`, `norm2`, `norm2b` (every
norm with `.b` and `.alpha`), `side.{gate,proj,norm}`; `mix.{q,k,v}` with `.conv`, `mix.{a,b,g,A_log,dt_bias,norm,o}` (delta);
`mix.{dq,dkv}` with `.norm`, `mix.{uq,uk,uv,g,o}` (latent attention); `mix.in`, `mix.conv` with `.b`,
`mix.{A_log,dt_bias,D,norm,o}` (mamba2); `mlp.table`, `mlp.e<j>.{gate,up,down}`.  Linear weights are [out, in].
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .kabanex import UNLIMITED_POSITIONS, _float, _get, _int
from .llama import ConfigError
from .specs import (
    ClampedExpertSpec,
    DynamicTanhSpec,
    EmbeddingSpec,
    GatedDeltaSpec,
    HeadSpec,
    LatentAttentionSpec,
    ModelSpec,
    NormSpec,
    RopeScalingSpec,
    RopeSpec,
    RoutedFeedForwardSpec,
    SandwichBlockSpec,
    ScheduleEntry,
    StateSpaceSpec,
    TokenSideSpec,
)

ARCHITECTURE = "Mabivik"
MIXERS = ("delta", "latent_attention", "mamba2")
# Constants the design fixes.
DELTA_UNIT_EPS = 1e-6  # unit vectors of the delta rule: x / sqrt(sum x^2 + 1e-6)
MAGNITUDE_SLOPE = 0.1  # stretched rotary tables are multiplied by 0.1 * ln(factor) + 1


@dataclass(frozen=True)
class MabivikDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class MabivikScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class MabivikLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int  # 0: no "mask", every earlier key is visible
    rot_base: float
    scaling: Optional[MabivikScaling]
    kv_from: Optional[int]


@dataclass(frozen=True)
class MabivikSpace:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int


@dataclass(frozen=True)
class MabivikExperts:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class MabivikLayer:
    type: str
    mixer: object
    mlp: Optional[MabivikExperts]


def _delta(mixer, where: str) -> MabivikDelta:
    heads, kv_heads = _int(mixer, "heads", where), _int(mixer, "kv_heads", where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}.heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    return MabivikDelta(heads, kv_heads, _int(mixer, "dim", where), _int(mixer, "vdim", where), _int(mixer, "conv", where))


def _latent(mixer, where: str, index: int) -> MabivikLatent:
    window = _int(mixer["mask"], "size", where + ".mask") if mixer.get("mask") is not None else 0
    rot_dim = _int(mixer, "rot_dim", where)
    rot = _get(mixer, "rot", where)
    rw = where + ".rot"
    if _int(rot, "dims", rw) != rot_dim or rot_dim % 2:
        raise ConfigError(f"config.json: {rw}.dims must be even and equal to rot_dim ({rot_dim}), got {rot['dims']}")
    base = _float(rot, "base", rw, positive=True)
    scaling = None
    if rot.get("scaling") is not None:
        if base == 1.0:
            raise ConfigError(f"config.json: {rw}.base must differ from 1")
        s, sw = rot["scaling"], rw + ".scaling"
        scaling = MabivikScaling(*(_float(s, key, sw, positive=True) for key in ("factor", "original", "fast", "slow")))
    kv_from = None
    if mixer.get("kv_from") is not None:
        kv_from = _int(mixer, "kv_from", where, least=0)
        if kv_from >= index:
            raise ConfigError(f"config.json: {where}.kv_from ({kv_from}) must name an earlier layer")
    return MabivikLatent(_int(mixer, "heads", where), _int(mixer, "dim", where), rot_dim, _int(mixer, "vdim", where),
                         _int(mixer, "q_rank", where), _int(mixer, "kv_rank", where), _float(mixer, "scale", where), window, base,
                         scaling, kv_from)


def _space(mixer, where: str) -> MabivikSpace:
    m = MabivikSpace(*(_int(mixer, key, where) for key in ("heads", "vdim", "state", "groups", "norm_groups", "conv")))
    if m.heads % m.groups:
        raise ConfigError(f"config.json: {where}.heads ({m.heads}) must be a multiple of groups ({m.groups})")
    if m.heads * m.vdim % m.norm_groups:
        raise ConfigError(f"config.json: {where}: {m.heads} heads of {m.vdim} do not form {m.norm_groups} equal parts")
    return m


def _feed_forward(mlp, where: str) -> Optional[MabivikExperts]:
    if mlp is None:
        return None
    if _get(mlp, "kind", where) != "moe":
        raise ConfigError(f"config.json: {where}.kind {mlp['kind']!r} is not built (known: moe)")
    router, rw = _get(mlp, "router", where), where + ".router"
    experts, top = _int(router, "experts", rw), _int(router, "top", rw)
    if top > experts:
        raise ConfigError(f"config.json: {rw}.top ({top}) exceeds the {experts} experts")
    return MabivikExperts(experts, top, _int(_get(mlp, "expert", where), "ff", where + ".expert"))


@dataclass(frozen=True)
class MabivikConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    side_dim: int  # 0: no "token_side"
    layers: Tuple[MabivikLayer, ...]

    @staticmethod
    def from_dict(raw: Mapping[str, Any]) -> "MabivikConfig":
        vocab = _int(raw, "vocab", "the model")
        width = _int(raw, "width", "the model")
        eps = _float(_get(raw, "norm", "the model"), "eps", "norm", positive=True)
        embedding_scale = _float(raw["embedding"], "scale", "embedding") if raw.get("embedding") is not None else 1.0
        logit_scale = _float(raw, "logit_scale", "the model") if raw.get("logit_scale") is not None else 1.0
        side = _int(raw["token_side"], "dim", "token_side") if raw.get("token_side") is not None else 0
        listed = _get(raw, "layers", "the model")
        if not isinstance(listed, (list, tuple)) or not listed:
            raise ConfigError("config.json: layers must be a non-empty list")
        layers = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]"
            kind = _get(entry, "type", where)
            mixer = _get(entry, "mixer", where)
            mw = where + ".mixer"
            if kind == "delta":
                parsed = _delta(mixer, mw)
            elif kind == "latent_attention":
                parsed = _latent(mixer, mw, i)
                if parsed.kv_from is not None:
                    source = layers[parsed.kv_from]
                    own = source.mixer if source.type == "latent_attention" and source.mixer.kv_from is None else None
                    if own is None:
                        raise ConfigError(f"config.json: {mw}.kv_from names layer {parsed.kv_from}, which makes no latent rows of its own")
                    if (own.kv_rank, own.rot_dim, own.rot_base, own.scaling) != (parsed.kv_rank, parsed.rot_dim, parsed.rot_base, parsed.scaling):
                        raise ConfigError(f"config.json: {mw} reads the rows of layer {parsed.kv_from}, whose kv_rank, rot_dim or rotation differs")
            elif kind == "mamba2":
                parsed = _space(mixer, mw)
            else:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not built (known: {', '.join(MIXERS)})")
            layers.append(MabivikLayer(kind, parsed, _feed_forward(entry.get("mlp"), where + ".mlp")))
        return MabivikConfig(str(raw.get("architecture", ARCHITECTURE)), vocab, width, eps, embedding_scale, logit_scale, side, tuple(layers))

    def to_dict(self) -> dict:
        layers = []
        for layer in self.layers:
            m = layer.mixer
            if layer.type == "delta":
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
            elif layer.type == "latent_attention":
                rot = {"dims": m.rot_dim, "base": m.rot_base}
                if m.scaling is not None:
                    s = m.scaling
                    rot["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
                mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
                         "scale": m.scale, "rot": rot}
                if m.window:
                    mixer["mask"] = {"size": m.window}
                if m.kv_from is not None:
                    mixer["kv_from"] = m.kv_from
            else:
                mixer = {"heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "norm_groups": m.norm_groups, "conv": m.conv}
            f = layer.mlp
            mlp = None if f is None else {"kind": "moe", "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.ff}}
            layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "embedding": {"scale": self.embedding_scale}, "logit_scale": self.logit_scale, "layers": layers}
        if self.side_dim:
            out["token_side"] = {"dim": self.side_dim}
        return out

    def _mixer_spec(self, layer: MabivikLayer, mp: str):
        m, W, eps = layer.mixer, self.width, self.norm_eps
        if layer.type == "delta":
            names = {r: mp + r for r in ("q", "k", "v", "o", "a", "b", "A_log", "dt_bias", "norm")}
            names.update(gate=mp + "g", q_conv=mp + "q.conv", k_conv=mp + "k.conv", v_conv=mp + "v.conv")
            return GatedDeltaSpec(hidden_size=W, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim,
                                  conv_taps=m.conv, unit_eps=DELTA_UNIT_EPS, eps=eps, weights=names)
        if layer.type == "latent_attention":
            names = {"down_q": mp + "dq", "down_q_norm": mp + "dq.norm", "up_q": mp + "uq", "down": mp + "dkv", "down_norm": mp + "dkv.norm",
                     "up_k": mp + "uk", "up_v": mp + "uv", "gate": mp + "g", "o": mp + "o"}
            s = m.scaling
            scaling = None if s is None else RopeScalingSpec("yarn", s.factor, low_freq_factor=s.slow, high_freq_factor=s.fast,
                                                             original_max_position=s.original,
                                                             magnitude=MAGNITUDE_SLOPE * math.log(s.factor) + 1.0)
            return LatentAttentionSpec(hidden_size=W, num_heads=m.heads, head_dim=m.dim, value_dim=m.vdim, latent_dim=m.kv_rank, scale=m.scale,
                                       eps=eps, gated=True, weights=names, query_latent=m.q_rank,
                                       position=RopeSpec(m.rot_dim, m.rot_base, "half", scaling), window=m.window or None,
                                       gate_kind="element", own_rows=m.kv_from is None)
        names = {r: mp + r for r in ("in", "conv", "A_log", "dt_bias", "D", "norm", "o")}
        names.update(conv_bias=mp + "conv.b")
        return StateSpaceSpec(hidden_size=W, num_heads=m.heads, value_dim=m.vdim, state_size=m.state, groups=m.groups,
                              norm_groups=m.norm_groups, conv_taps=m.conv, eps=eps, weights=names)

    def model_spec(self) -> ModelSpec:
        W, eps, count = self.width, self.norm_eps, len(self.layers)
        norm = lambda name: DynamicTanhSpec(W, {"weight": name, "bias": name + ".b", "alpha": name + ".alpha"})  # noqa: E731
        blocks = []
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            parts = dict(mixer=self._mixer_spec(layer, p + "mix."), mixer_norm=norm(p + "norm1"), mixer_out_norm=norm(p + "norm1b"))
            f = layer.mlp
            if f is not None:
                names = {"table": p + "mlp.table", **{"expert_" + r: p + "mlp.e{expert}." + r for r in ("gate", "up", "down")}}
                plain = ClampedExpertSpec(f.ff, math.inf, 1.0, up_offset=0.0)  # silu(gate) * up
                parts.update(feed_forward=RoutedFeedForwardSpec(hidden_size=W, num_experts=f.experts, top=f.top, expert=plain, shared=None,
                                                                weights=names, rule="table", vocab_size=self.vocab),
                             feed_forward_norm=norm(p + "norm2"), feed_forward_out_norm=norm(p + "norm2b"))
            if self.side_dim:
                parts.update(side=TokenSideSpec(W, self.vocab, self.side_dim, i, count,
                                                {"table": "side.embed", "gate": p + "side.gate", "proj": p + "side.proj"}),
                             side_norm=NormSpec(W, eps, {"weight": p + "side.norm"}))
            blocks.append(SandwichBlockSpec(**parts))
        # a layer without a feed-forward reads no norms around it; a file that holds them all the same is taken
        unused = tuple(f"l{i}.{name}{tail}" for i, layer in enumerate(self.layers) if layer.mlp is None
                       for name in ("norm2", "norm2b") for tail in ("", ".b", ".alpha"))
        sources = [layer.mixer.kv_from if layer.type == "latent_attention" else None for layer in self.layers]
        return ModelSpec(
            architecture=self.architecture,
            vocab_size=self.vocab,
            hidden_size=W,
            max_positions=UNLIMITED_POSITIONS,
            embedding=EmbeddingSpec(self.vocab, W, self.embedding_scale, {"weight": "embed"}),
            layers=tuple(blocks),
            schedule=tuple(ScheduleEntry(i, cache_from=source) for i, source in enumerate(sources)),
            final_norm=norm("final.norm"),
            head=HeadSpec(self.vocab, W, False, {"weight": "head"}, logit_scale=self.logit_scale),
            ignored_tensors=unused,
        )
