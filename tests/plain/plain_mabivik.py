"""A plain, slow Mabivik in float64: whole sequences, no cache, one function per mechanism.

It shares nothing with the package: it reads a configuration dictionary (the keys of the design's config.json) and a
dictionary of tensors by their checkpoint names, and walks every recurrence token by token.

The design.  x_0 = E[token] * embedding.scale.  With N a dynamic tanh, N(x) = tanh(alpha x) w + b, layer i runs
x += N1b(mixer(N1(x))); x += N2b(ff(N2(x))) (if it has a feed-forward); and then lets the token itself in once more:
x += rms(P (gelu_tanh(G x) * e)) with e the layer's columns of a second table's row.  Mixers: a gated delta rule, an
attention over a latent row and one shared rotated key (with a window; a layer may read the rows another layer cached),
a state-space recurrence with one decay per head and token.  Feed-forward: experts chosen by a table of token ids, weights
1 / top.  Logits = H N(x) * logit_scale.
"""

from __future__ import annotations

import math

import torch

from .plain_llama import read_model_folder  # noqa: F401  (reads config.json and the safetensors file)

F = torch.float64
DELTA_UNIT_EPS = 1e-6  # the delta rule's unit vectors: x / sqrt(sum x^2 + 1e-6)


def f64(t):
    return t.to(F)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def over_rms(x, eps):
    """Over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def dynamic_tanh(x, w, name):
    return torch.tanh(f64(w[name + ".alpha"]) * x) * f64(w[name]) + f64(w[name + ".b"])


def causal_conv(x, taps_w, bias=None):
    """x [T, C], taps_w [C, taps] whose last column meets the current token; zeros before the start."""
    T, C = x.shape
    taps = taps_w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=F), x], dim=0)
    out = torch.zeros(T, C, dtype=F)
    for i in range(taps):
        out += padded[i:i + T] * taps_w[:, i][None, :]
    return out if bias is None else out + bias


def gated_delta_rule(h, w, name, c, eps):
    """Per head: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    T = h.shape[0]
    H, G, D, Dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = silu(causal_conv(h @ f64(w[name + "q"]).T, f64(w[name + "q.conv"]))).view(T, G, D)
    k = silu(causal_conv(h @ f64(w[name + "k"]).T, f64(w[name + "k.conv"]))).view(T, G, D)
    v = silu(causal_conv(h @ f64(w[name + "v"]).T, f64(w[name + "v.conv"]))).view(T, H, Dv)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + DELTA_UNIT_EPS) * D ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + DELTA_UNIT_EPS)
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)  # head h uses q/k head h // (H / G)
    beta = torch.sigmoid(h @ f64(w[name + "b"]).T)
    decay = torch.exp(-torch.exp(f64(w[name + "A_log"])) * softplus(h @ f64(w[name + "a"]).T + f64(w[name + "dt_bias"])))
    gate = silu(h @ f64(w[name + "g"]).T).view(T, H, Dv)
    S = torch.zeros(H, D, Dv, dtype=F)
    out = torch.zeros(T, H, Dv, dtype=F)
    for t in range(T):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    out = over_rms(out, eps) * f64(w[name + "norm"]) * gate
    return out.reshape(T, H * Dv) @ f64(w[name + "o"]).T


def stretched_frequencies(rot):
    """The pairs' turns per position; with `scaling`, slow pairs are divided by its factor and fast ones kept."""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if s is None:
        return plain, 1.0

    def pair(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(pair(s["fast"])), 0), min(math.ceil(pair(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_half(x, positions, rot):
    """x [T, heads, dims]: coordinate i pairs with i + dims/2."""
    frequencies, magnitude = stretched_frequencies(rot)
    half = rot["dims"] // 2
    angle = positions.to(F)[:, None] * torch.tensor(frequencies, dtype=F)[None, :]
    c, s = (torch.cos(angle) * magnitude)[:, None, :], (torch.sin(angle) * magnitude)[:, None, :]
    a, b = x[..., :half], x[..., half:rot["dims"]]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., rot["dims"]:]], dim=-1)


def window_visible(T, size):
    """[T, T] booleans: query i sees key j when 0 <= i - j < size (None: every earlier key)."""
    p = torch.arange(T)
    behind = p[:, None] - p[None, :]
    seen = behind >= 0
    return seen if size is None else seen & (behind < size)


def latent_rows(h, w, name, c, eps):
    """What a layer caches per position: the normed latent and the rotated key part all heads share."""
    row = h @ f64(w[name + "dkv"]).T
    latent = over_rms(row[:, :c["kv_rank"]], eps) * f64(w[name + "dkv.norm"])
    rotated = rotate_half(row[:, None, c["kv_rank"]:], torch.arange(h.shape[0]), c["rot"])[:, 0]
    return latent, rotated


def latent_attention(h, w, name, c, eps, rows):
    """`rows`: this layer's latent_rows, or those of the layer named by kv_from."""
    T = h.shape[0]
    H, D, R, Dv = c["heads"], c["dim"], c["rot_dim"], c["vdim"]
    latent, rotated = rows
    q = (over_rms(h @ f64(w[name + "dq"]).T, eps) * f64(w[name + "dq.norm"])) @ f64(w[name + "uq"]).T
    q = q.view(T, H, D + R)
    q_rot = rotate_half(q[..., D:], torch.arange(T), c["rot"])
    k = (latent @ f64(w[name + "uk"]).T).view(T, H, D)
    v = (latent @ f64(w[name + "uv"]).T).view(T, H, Dv)
    seen = window_visible(T, c["mask"]["size"] if c.get("mask") else None)
    out = torch.zeros(T, H, Dv, dtype=F)
    for head in range(H):
        score = (q[:, head, :D] @ k[:, head].T + q_rot[:, head] @ rotated.T) * c["scale"]
        out[:, head] = torch.softmax(score.masked_fill(~seen, float("-inf")), dim=-1) @ v[:, head]
    out = out.reshape(T, H * Dv) * torch.sigmoid(h @ f64(w[name + "g"]).T)
    return out @ f64(w[name + "o"]).T


def state_space(h, w, name, c, eps):
    """Per head: S <- exp(-exp(A_log) dt) S + dt B x^T; y = S^T C + D x."""
    T = h.shape[0]
    H, P, N, G = c["heads"], c["vdim"], c["state"], c["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ f64(w[name + "in"]).T, [inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(causal_conv(xbc, f64(w[name + "conv"]), f64(w[name + "conv.b"])))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    x = x.view(T, H, P)
    B = B.view(T, G, N).repeat_interleave(H // G, dim=1)  # head h uses group h // (H / G)
    C = C.view(T, G, N).repeat_interleave(H // G, dim=1)
    dt = softplus(dt + f64(w[name + "dt_bias"]))
    decay = torch.exp(-torch.exp(f64(w[name + "A_log"])) * dt)
    S = torch.zeros(H, N, P, dtype=F)
    y = torch.zeros(T, H, P, dtype=F)
    for t in range(T):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnp,hn->hp", S, C[t]) + f64(w[name + "D"])[:, None] * x[t]
    y = y.reshape(T, inner) * silu(z)  # the gate comes before the norm
    parts = c["norm_groups"]
    y = over_rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * f64(w[name + "norm"])
    return y @ f64(w[name + "o"]).T


def table_experts(h, w, name, c, tokens):
    """Every token id's row of the table names its experts; each counts 1 / top."""
    top = c["router"]["top"]
    out = torch.zeros_like(h)
    for t, token in enumerate(tokens):
        for e in w[name + "table"][token].tolist():
            p = f"{name}e{int(e)}."
            x = h[t]
            out[t] += f64(w[p + "down"]) @ (silu(f64(w[p + "gate"]) @ x) * (f64(w[p + "up"]) @ x)) / top
    return out


def token_side(x, w, layer, dim, index, tokens, eps):
    e = f64(w["side.embed"])[torch.as_tensor(tokens, dtype=torch.long), index * dim:(index + 1) * dim]
    y = (gelu_tanh(x @ f64(w[layer + "side.gate"]).T) * e) @ f64(w[layer + "side.proj"]).T
    return over_rms(y, eps) * f64(w[layer + "side.norm"])


def forward(config, w, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence (and, if asked, the stream after every layer [layers, T, W])."""
    eps = config["norm"]["eps"]
    tokens = [int(t) for t in tokens]
    x = f64(w["embed"])[torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    layers, cached = [], {}
    for i, layer in enumerate(config["layers"]):
        p, c = f"l{i}.", layer["mixer"]
        h = dynamic_tanh(x, w, p + "norm1")
        if layer["type"] == "delta":
            m = gated_delta_rule(h, w, p + "mix.", c, eps)
        elif layer["type"] == "latent_attention":
            if c.get("kv_from") is None:
                cached[i] = latent_rows(h, w, p + "mix.", c, eps)
            m = latent_attention(h, w, p + "mix.", c, eps, cached[i if c.get("kv_from") is None else c["kv_from"]])
        elif layer["type"] == "mamba2":
            m = state_space(h, w, p + "mix.", c, eps)
        else:
            raise ValueError(layer["type"])
        x = x + dynamic_tanh(m, w, p + "norm1b")
        if layer.get("mlp") is not None:
            f = table_experts(dynamic_tanh(x, w, p + "norm2"), w, p + "mlp.", layer["mlp"], tokens)
            x = x + dynamic_tanh(f, w, p + "norm2b")
        if config.get("token_side") is not None:
            x = x + token_side(x, w, p, config["token_side"]["dim"], i, tokens, eps)
        layers.append(x.clone())
    logits = dynamic_tanh(x, w, "final.norm") @ f64(w["head"]).T * config["logit_scale"]
    return (logits, torch.stack(layers)) if return_layers else logits
