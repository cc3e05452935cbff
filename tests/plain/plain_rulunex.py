"""A plain, slow Rulunex in float64: whole sequences, no cache, one function per mechanism.

It shares nothing with the package: it reads a configuration dictionary (the keys of the design's config.json) and a
dictionary of tensors by their checkpoint names.

The design.  x_0 = E[token] * embedding.scale.  A layer has one norm, N(x) = x / rms(x) * (1 + w), whose rows both sublayers read:
x += mixer(N(x)) + ff(N(x)) (or the mixer alone).  A span of layers runs several times in a row with the same weights; ahead of
every pass the stream is made anew from itself and the embedding's rows, x <- J [x; x_0].  Mixers: an attention over an RMS-normed
latent row and one rotated key part that all heads share, with a gate per head; a windowed grouped-query attention whose values are
its projected keys and whose queries and keys pass one RMS norm each over the whole projection.  The feed-forward is gated, with
both branches clamped.  Logits = E N(x).
"""

from __future__ import annotations

import math

import torch

from .plain_llama import read_model_folder  # noqa: F401  (reads config.json and the safetensors file)

F = torch.float64
SWISH_SLOPE = 1.702


def f64(t):
    return t.to(F)


def over_rms(x, eps):
    """Over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_one(x, w, name, eps):
    return over_rms(x, eps) * (1.0 + f64(w[name]))


def turns(rot):
    """The pairs' turns per position; with `scaling`, pairs of long wavelengths turn more slowly."""
    out = []
    for i in range(rot["dims"] // 2):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s is not None:
            length = 2.0 * math.pi / f
            if length > s["original"] / s["low"]:
                f = f / s["factor"]
            elif length >= s["original"] / s["high"]:
                share = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - share) * f / s["factor"] + share * f
        out.append(f)
    return torch.tensor(out, dtype=F)


def _angles(T, rot):
    a = torch.arange(T).to(F)[:, None] * turns(rot)[None, :]
    return torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]


def rotate_half(x, rot):
    """x [T, heads, size]: coordinate i pairs with i + dims/2; what lies behind `dims` stays."""
    n, half = rot["dims"], rot["dims"] // 2
    c, s = _angles(x.shape[0], rot)
    u, v = x[..., :half], x[..., half:n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], dim=-1)


def rotate_neighbours(x, rot):
    """x [T, heads, size]: coordinate 2i pairs with 2i + 1; what lies behind `dims` stays."""
    n = rot["dims"]
    c, s = _angles(x.shape[0], rot)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2)
    return torch.cat([turned, x[..., n:]], dim=-1)


def window_visible(T, size):
    """[T, T] booleans: query i sees key j when 0 <= i - j < size (None: every earlier key)."""
    p = torch.arange(T)
    behind = p[:, None] - p[None, :]
    seen = behind >= 0
    return seen if size is None else seen & (behind < size)


def softmax_sum(score, seen, v):
    return torch.softmax(score.masked_fill(~seen, float("-inf")), dim=-1) @ v


def latent_attention(h, w, name, c, eps):
    T = h.shape[0]
    H, D, R, Dv, rank = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    q = (h @ f64(w[name + "q"]).T).view(T, H, D + R)
    row = h @ f64(w[name + "dkv"]).T
    latent = over_rms(row[:, :rank], eps) * f64(w[name + "dkv.norm"])
    q_rot, k_rot = rotate_neighbours(q[..., D:], c["rot"]), rotate_neighbours(row[:, None, rank:], c["rot"])[:, 0]
    k = (latent @ f64(w[name + "uk"]).T).view(T, H, D)
    v = (latent @ f64(w[name + "uv"]).T).view(T, H, Dv)
    gate = torch.sigmoid(h @ f64(w[name + "g"]).T)
    seen = window_visible(T, None)
    out = torch.zeros(T, H, Dv, dtype=F)
    for head in range(H):
        score = (q[:, head, :D] @ k[:, head].T + q_rot[:, head] @ k_rot.T) * c["scale"]
        out[:, head] = softmax_sum(score, seen, v[:, head]) * gate[:, head:head + 1]
    return out.reshape(T, H * Dv) @ f64(w[name + "o"]).T


def attention(h, w, name, c, eps):
    T = h.shape[0]
    H, G, D = c["heads"], c["kv_heads"], c["dim"]
    q, k = h @ f64(w[name + "q"]).T, h @ f64(w[name + "k"]).T
    v = k.view(T, G, D)  # the keys as projected
    q = (over_rms(q, eps) * f64(w[name + "q.norm"])).view(T, H, D)
    k = (over_rms(k, eps) * f64(w[name + "k.norm"])).view(T, G, D)
    if c.get("rot") is not None:
        q, k = rotate_half(q, c["rot"]), rotate_half(k, c["rot"])
    seen = window_visible(T, c["mask"]["size"] if c.get("mask") else None)
    out = torch.zeros(T, H, D, dtype=F)
    for head in range(H):
        g = head // (H // G)
        out[:, head] = softmax_sum(q[:, head] @ k[:, g].T * c["scale"], seen, v[:, g])
    return out.reshape(T, H * D) @ f64(w[name + "o"]).T


def clamped_feed_forward(h, w, name, c):
    g = torch.clamp(h @ f64(w[name + "gate"]).T, max=c["limit"])
    u = torch.clamp(h @ f64(w[name + "up"]).T, min=-c["limit"], max=c["limit"])
    return (g * torch.sigmoid(SWISH_SLOPE * g) * (u + 1.0)) @ f64(w[name + "down"]).T


def join(x, x0, w):
    return torch.cat([x, x0], dim=-1) @ f64(w["loop.in"]).T


def run_order(config):
    """(layer, whether a pass begins with it) for every run."""
    n, loop = len(config["layers"]), config.get("loop")
    if loop is None:
        return [(i, False) for i in range(n)]
    span = [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return [(i, False) for i in range(loop["start"])] + span * loop["times"] + [(i, False) for i in range(loop["stop"], n)]


MIXERS = {"latent_attention": latent_attention, "attention": attention}


def forward(config, w, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence (and, if asked, the stream after every layer run [runs, T, W])."""
    eps = config["norm"]["eps"]
    x0 = f64(w["embed"])[torch.as_tensor([int(t) for t in tokens], dtype=torch.long)] * config["embedding"]["scale"]
    x, layers = x0, []
    for i, begins in run_order(config):
        layer, p = config["layers"][i], f"l{i}."
        if begins:
            x = join(x, x0, w)
        h = norm_around_one(x, w, p + "norm1", eps)
        y = MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + clamped_feed_forward(h, w, p + "mlp.", layer["mlp"])
        x = x + y
        layers.append(x.clone())
    logits = norm_around_one(x, w, "final.norm", eps) @ f64(w["embed"]).T
    return (logits, torch.stack(layers)) if return_layers else logits
