"""Small Mabivik configurations for the tests.  They differ from one another in every size and constant, and between their own
layers: the order of the mixers, head counts (one head, as many query/key heads as heads, one, others), key, rotated, value and
latent sizes (equal, unequal, no multiples of 8), windows of 1, of 5, of 64, of 100 and none, attentions that read another layer's
rows with a narrower, a wider and no window, 1 to 5 convolution weights, one group and several, norm parts that cut through heads,
one expert per token and many, layers without a feed-forward, scales of 1 and others, and widths the tensor-core products do not
take."""

from __future__ import annotations

from pathlib import Path

import torch

from plain import plain_mabivik


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def delta(heads, kv_heads, dim, vdim, taps, mlp):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window, rot, mlp, kv_from=None):
    """rot: (base, (factor, original, fast, slow) or None)."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"dims": rot_dim, "base": rot[0]}}
    if rot[1] is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[1]))
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def mamba2(heads, vdim, state, groups, norm_groups, taps, mlp):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups,
                                        "conv": taps}, "mlp": mlp}


def model(vocab, width, eps, embedding_scale, logit_scale, side, layers):
    return {"architecture": "Mabivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embedding_scale},
            "logit_scale": logit_scale, "token_side": {"dim": side}, "layers": layers}


ROT_A, ROT_B, ROT_C = (10000.0, (4.0, 64.0, 8.0, 1.0)), (500.0, None), (100000.0, (1.5, 300.0, 16.0, 2.0))

MBV_A = model(210, 64, 1e-5, 2.0, 0.25, 12, [
    mamba2(4, 16, 24, 2, 2, 3, moe(6, 2, 40)),
    latent(4, 16, 8, 8, 24, 32, 0.3, 5, ROT_A, moe(4, 1, 24)),
    delta(2, 1, 16, 24, 4, None),
    latent(2, 24, 8, 16, 40, 32, 0.2, 70, ROT_A, moe(3, 3, 20), kv_from=1),   # a wider window than the rows' owner
    mamba2(3, 8, 8, 1, 4, 2, moe(5, 2, 16)),                                  # parts of 6 numbers cut through heads of 8
])

MBV_B = model(150, 72, 1e-6, 1.0, 1.0, 8, [
    latent(3, 20, 10, 12, 33, 22, 0.22, 100, ROT_B, moe(5, 3, 36)),
    delta(4, 4, 12, 6, 5, moe(2, 1, 20)),
    latent(1, 8, 10, 40, 16, 22, 0.35, None, ROT_B, None, kv_from=0),         # no window at all over a windowed layer's rows
    latent(3, 16, 4, 10, 20, 16, 0.3, 1, ROT_C, moe(3, 2, 20)),               # a window of one position
    mamba2(1, 32, 32, 1, 1, 1, moe(4, 4, 12)),
])

# sizes at which the tensor-core products, the tensor-core attention and the state-space chunks run
MBV_C = model(512, 256, 1e-5, 0.7, 0.5, 40, [
    delta(4, 2, 64, 128, 4, moe(8, 2, 128)),
    latent(8, 32, 16, 48, 96, 112, 0.144, 64, ROT_C, moe(4, 1, 64)),
    mamba2(6, 32, 64, 3, 3, 4, moe(8, 3, 64)),
    latent(4, 64, 16, 32, 64, 112, 0.11, 33, ROT_C, moe(4, 2, 64), kv_from=1),
])

# a width and head sizes that are no multiples of 8
MBV_D = model(131, 50, 3e-6, 1.3, 2.0, 7, [
    delta(6, 2, 18, 10, 3, moe(5, 2, 33)),
    mamba2(5, 6, 18, 5, 3, 2, moe(7, 3, 12)),
    latent(6, 10, 6, 14, 21, 26, 0.24, 7, (50.0, (2.0, 40.0, 4.0, 0.5)), None),
    latent(1, 6, 6, 3, 9, 26, 0.4, 33, (50.0, (2.0, 40.0, 4.0, 0.5)), moe(2, 2, 10), kv_from=2),
])

MBV = {"A": MBV_A, "B": MBV_B, "C": MBV_C, "D": MBV_D}


def make_folder(raw: dict, seed: int, root) -> Path:
    """A folder with random weights.  Some tensors are then drawn anew so that they matter: convolution weights of both signs and of
    size one, recurrences that forget slowly and quickly (so that a lost state shows), dynamic tanhs away from their straight middle,
    sharp attention scores, tables that use every expert."""
    from models_b200.config import config_from_dict
    from models_b200.weights import write_random_model
    from models_b200.weights.safetensors_io import write_safetensors

    folder = Path(root) / f"mabivik_{seed}"
    write_random_model(folder, config_from_dict(raw), seed, std=1.1 * raw["width"] ** -0.5, gain_std=0.1, dtype=torch.bfloat16)
    _, weights = plain_mabivik.read_model_folder(folder)
    g = torch.Generator().manual_seed(seed)
    for name in list(weights):
        shape = weights[name].shape
        uniform = lambda lo, hi: torch.rand(shape, generator=g) * (hi - lo) + lo  # noqa: E731
        if name.endswith(".conv"):
            t = torch.randn(shape, generator=g) * 0.6
        elif name.endswith(".conv.b"):
            t = torch.randn(shape, generator=g) * 0.3
        elif name.endswith(".A_log"):
            t = uniform(-3.0, 0.5)
        elif name.endswith(".dt_bias"):
            t = uniform(-2.0, 1.0)
        elif name.endswith(".D"):
            t = uniform(-1.0, 1.5)
        elif name.endswith(".alpha"):
            t = uniform(0.4, 1.2)
        elif name.endswith(("norm1.b", "norm2.b", "norm1b.b", "norm2b.b", "final.norm.b")):
            t = torch.randn(shape, generator=g) * 0.1
        elif name.endswith((".mix.a", ".mix.b")):
            t = torch.randn(shape, generator=g) * (4 * shape[1] ** -0.5)
        elif name.endswith((".uq", ".uk")):
            t = torch.randn(shape, generator=g) * (1.6 * shape[1] ** -0.5)
        elif name in ("embed", "side.embed"):
            t = torch.randn(shape, generator=g) * 0.6
        elif name.endswith(".mlp.table"):
            experts = next(layer for i, layer in enumerate(raw["layers"]) if name.startswith(f"l{i}."))["mlp"]["router"]["experts"]
            weights[name] = torch.stack([torch.randperm(experts, generator=g)[:shape[1]] for _ in range(shape[0])]).to(torch.int32)
            continue
        else:
            continue
        weights[name] = t.to(torch.bfloat16)
    write_safetensors(folder / "model.safetensors", {n: t.contiguous() for n, t in weights.items()}, {"format": "pt"})
    return folder


def plain_logits(folder, tokens, layers_out=None) -> torch.Tensor:
    config, weights = plain_mabivik.read_model_folder(folder)
    if layers_out is None:
        return plain_mabivik.forward(config, weights, list(tokens))
    logits, layers = plain_mabivik.forward(config, weights, list(tokens), return_layers=True)
    layers_out.extend(layers)
    return logits
