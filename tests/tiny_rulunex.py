"""Small Rulunex configurations for the tests.  They differ from one another in every size and constant, and between their own
layers: the order of the mixers, head counts (one head, as many key/value heads as heads, one, others), key, rotated, value and
latent sizes (equal, unequal, no multiples of 8), windows of 1, of 5, of 64, of 100 and none, whole heads rotated, parts of them
and none, stretched frequencies with pairs on both sides and in between, layers without a feed-forward, limits that cut much and
little, loops over the first layers, the last ones, all of them, one pass, three passes and none, and widths the tensor-core products
do not take."""

from __future__ import annotations

from pathlib import Path

import torch

from plain import plain_rulunex


def attention(heads, kv_heads, dim, scale, window, rot, ff, limit=1.0):
    """rot: None or (dims, base, (factor, low, high, original) or None); ff 0: no feed-forward."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if rot[2] is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), rot[2]))
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, ff, limit=1.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"dims": rot_dim, "base": base}}
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def model(vocab, width, eps, embedding_scale, loop, layers):
    """loop: None or (start, stop, times)."""
    out = {"architecture": "Rulunex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embedding_scale}, "layers": layers}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


STRETCHED = (8.0, 1.0, 4.0, 48)

RLX_A = model(210, 64, 1e-5, 2.0, (1, 3, 3), [
    latent(4, 16, 8, 8, 32, 0.3, 10000.0, 40, 0.5),
    attention(4, 2, 16, 0.3, 5, (8, 500.0, STRETCHED), 24, 3.0),
    latent(2, 8, 16, 24, 48, 0.25, 50.0, 0),
    attention(2, 1, 24, 0.2, None, (24, 10000.0, (2.0, 0.5, 8.0, 100)), 32, 0.8),
])

RLX_B = model(150, 72, 1e-6, 1.0, (0, 2, 2), [
    attention(3, 3, 20, 0.25, 100, (10, 1000.0, None), 36, 1.5),
    attention(6, 2, 12, 0.3, 1, None, 0),                            # a window of one position, nothing rotated
    latent(1, 40, 10, 12, 22, 0.22, 5000.0, 20, 0.3),
])

# sizes at which the tensor-core products and the tensor-core attention run; every layer in the loop, one pass
RLX_C = model(512, 256, 1e-5, 0.7, (0, 4, 1), [
    latent(8, 32, 16, 48, 112, 0.144, 20000.0, 192, 2.0),
    attention(8, 4, 32, 0.18, 64, (32, 20000.0, STRETCHED), 128, 0.7),
    latent(16, 48, 16, 16, 64, 0.125, 300.0, 256, 1.2),
    attention(4, 1, 64, 0.125, 33, (16, 20000.0, None), 0),
])

# a width, head sizes and feed-forwards that are no multiples of 8; the last layers in the loop
RLX_D = model(131, 50, 3e-6, 1.3, (2, 4, 2), [
    attention(5, 5, 10, 0.35, 7, (6, 100.0, (3.0, 1.0, 2.0, 30)), 33, 0.6),
    latent(6, 10, 6, 14, 26, 0.24, 50.0, 0),
    attention(2, 1, 14, 0.3, 70, (14, 100.0, None), 18, 5.0),
    latent(1, 6, 2, 3, 9, 0.4, 900.0, 27, 1.1),
])

# no loop at all
RLX_E = model(90, 128, 1e-5, 3.0, None, [
    latent(2, 64, 64, 128, 64, 0.09, 20000.0, 96, 1.0),
    attention(4, 2, 32, 0.2, 64, (16, 2000.0, STRETCHED), 64, 1.0),
])

RLX = {"A": RLX_A, "B": RLX_B, "C": RLX_C, "D": RLX_D, "E": RLX_E}


def make_folder(raw: dict, seed: int, root) -> Path:
    """A folder with random weights.  Some tensors are drawn anew so that they matter: layer norms well away from one, sharp attention
    scores, feed-forward branches that reach their limits, a join whose two halves weigh the same."""
    from models_b200.config import config_from_dict
    from models_b200.weights import write_random_model
    from models_b200.weights.safetensors_io import write_safetensors

    folder = Path(root) / f"rulunex_{seed}"
    write_random_model(folder, config_from_dict(raw), seed, std=1.1 * raw["width"] ** -0.5, gain_std=0.1, dtype=torch.bfloat16)
    _, weights = plain_rulunex.read_model_folder(folder)
    g = torch.Generator().manual_seed(seed)
    for name in list(weights):
        shape = weights[name].shape
        if name.endswith(".norm1") or name == "final.norm":
            t = torch.randn(shape, generator=g) * 0.35
        elif name.endswith((".q.norm", ".k.norm")):
            t = 1.3 + torch.randn(shape, generator=g) * 0.3
        elif name.endswith((".uk", ".mix.q", ".mix.k")):
            t = torch.randn(shape, generator=g) * (1.6 * shape[1] ** -0.5)
        elif name == "loop.in":
            t = torch.randn(shape, generator=g) * (shape[1] ** -0.5)
        elif name == "embed":
            t = torch.randn(shape, generator=g) * 0.6
        else:
            continue
        weights[name] = t.to(torch.bfloat16)
    write_safetensors(folder / "model.safetensors", {n: t.contiguous() for n, t in weights.items()}, {"format": "pt"})
    return folder


def plain_logits(folder, tokens, layers_out=None) -> torch.Tensor:
    config, weights = plain_rulunex.read_model_folder(folder)
    if layers_out is None:
        return plain_rulunex.forward(config, weights, list(tokens))
    logits, layers = plain_rulunex.forward(config, weights, list(tokens), return_layers=True)
    layers_out.extend(layers)
    return logits
