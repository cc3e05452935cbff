"""Rulunex without a GPU: the configuration reader (round trip, refusals, the tensors a model asks for), the schedule with its joins,
the cache groups of a looped model, the order in which rotated rows are loaded, and the plain implementation against cases worked out
by hand, against itself, and against mistakes planted in it (which the tests' models must show)."""

import copy
import math

import pytest
import torch

from plain import plain_rulunex as pr
from tiny import TOLERANCE, random_tokens, scaled_error
from tiny_rulunex import RLX, STRETCHED, attention, latent, make_folder, model, plain_logits

F = torch.float64


@pytest.mark.parametrize("name", sorted(RLX))
def test_configuration_round_trip_and_tensors(name):
    from models_b200.config import config_from_dict
    from models_b200.engine.model import parameter_requests

    raw = RLX[name]
    config = config_from_dict(raw)
    assert config.to_dict() == raw
    spec = config.model_spec()
    assert spec.head.tied and spec.head.logit_scale == 1.0 and spec.embedding.scale == raw["embedding"]["scale"]
    assert [(e.layer, e.joins) for e in spec.schedule] == pr.run_order(raw)
    W = raw["width"]
    requests = parameter_requests(spec)
    expected = {"embed": (raw["vocab"], W), "final.norm": (W,)}
    if raw.get("loop"):
        expected["loop.in"] = (W, 2 * W)
    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        expected[p + "norm1"] = (W,)
        if layer["type"] == "attention":
            q, k = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
            expected.update({p + "mix.q": (q, W), p + "mix.k": (k, W), p + "mix.q.norm": (q,), p + "mix.k.norm": (k,), p + "mix.o": (W, q)})
        else:
            H, K = m["heads"], m["kv_rank"]
            expected.update({p + "mix.q": (H * (m["dim"] + m["rot_dim"]), W), p + "mix.dkv": (K + m["rot_dim"], W), p + "mix.dkv.norm": (K,),
                             p + "mix.uk": (H * m["dim"], K), p + "mix.uv": (H * m["vdim"], K), p + "mix.g": (H, W), p + "mix.o": (W, H * m["vdim"])})
        if layer["mlp"]:
            f = layer["mlp"]["ff"]
            expected.update({p + "mlp.gate": (f, W), p + "mlp.up": (f, W), p + "mlp.down": (W, f)})
    assert {n: tuple(r.shape) for n, r in requests.items()} == expected


def test_configurations_that_are_refused():
    from models_b200.config import ConfigError, config_from_dict

    good = model(50, 16, 1e-5, 1.0, (0, 1, 2), [attention(2, 1, 8, 0.3, 5, (4, 100.0, STRETCHED), 8), latent(2, 8, 4, 8, 8, 0.3, 100.0, 8)])
    config_from_dict(good)

    def refused(change):
        bad = copy.deepcopy(good)
        change(bad)
        with pytest.raises(ConfigError):
            config_from_dict(bad)

    a, b = (lambda c: c["layers"][0]["mixer"]), (lambda c: c["layers"][1]["mixer"])
    for change in (lambda c: c["layers"][0].update(type="mamba2"), lambda c: a(c).update(vdim=6), lambda c: a(c).update(kv_heads=3),
                   lambda c: a(c)["rot"].update(dims=10), lambda c: a(c)["rot"].update(dims=3), lambda c: a(c)["mask"].update(size=0),
                   lambda c: a(c)["rot"]["scaling"].update(low=4.0), lambda c: a(c)["rot"]["scaling"].pop("original"), lambda c: a(c).pop("scale"),
                   lambda c: b(c)["rot"].update(dims=8), lambda c: b(c).update(rot_dim=3), lambda c: b(c).pop("kv_rank"),
                   lambda c: c["layers"][1]["mlp"].update(kind="moe"), lambda c: c["layers"][1]["mlp"].update(limit=0.0),
                   lambda c: c["loop"].update(stop=3), lambda c: c["loop"].update(start=1), lambda c: c["loop"].update(times=0),
                   lambda c: c.update(layers=[]), lambda c: c["norm"].update(eps=0.0)):
        refused(change)


def test_a_join_needs_a_part_and_one_stream():
    from dataclasses import replace

    from models_b200.config import config_from_dict

    spec = config_from_dict(RLX["A"]).model_spec()
    for change in ({"join": None}, {"residual_streams": 2}):
        with pytest.raises(ValueError):
            replace(spec, **change)


def test_cache_groups_of_a_looped_model():
    """Every pass of a looped layer owns rows of its own; layers that need the same share a group; windows are kept apart."""
    from models_b200.cache.kv_cache import KvCache
    from models_b200.config import config_from_dict
    from models_b200.engine.model import DecoderModel
    from models_b200.parts import Runtime

    raw = model(50, 32, 1e-5, 1.0, (0, 2, 3), [attention(2, 1, 16, 0.3, 70, (4, 100.0, None), 8), latent(2, 8, 4, 8, 12, 0.3, 100.0, 8),
                                               attention(4, 1, 16, 0.3, None, None, 0)])
    spec = config_from_dict(raw).model_spec()
    decoder = DecoderModel(spec, Runtime(torch.device("meta"), "float32", max_positions=1))
    requests = decoder.kv_requests()
    assert [(r.num_kv_heads, r.head_dim, r.window, r.value_dim) for r in requests] == [(1, 16, 70, 16), (1, 16, None, 0)] * 3 + [(1, 16, None, 16)]
    cache = KvCache(requests, [e.cache_from for e in spec.schedule], 256, 4, 64, None)
    assert len({(cache.run_location[r]) for r in range(7)}) == 7
    assert sorted(len(g.runs) for g in cache.groups) == [1, 3, 3]


@pytest.mark.parametrize("rot_dim", [2, 6, 16])
def test_rotated_rows_are_loaded_as_pairs_of_halves(rot_dim):
    """A latent attention whose spec pairs neighbours: its matrices come out with the even coordinates of a rotated part first."""
    from models_b200.config import config_from_dict
    from models_b200.parts import Runtime, build_part

    H, D, K = 3, 5, 7
    raw = model(50, 4, 1e-5, 1.0, None, [latent(H, D, rot_dim, 4, K, 0.3, 100.0, 0)])
    part = build_part("mixer", config_from_dict(raw).model_spec().layers[0].mixer, Runtime(torch.device("cpu"), "float32", max_positions=4))
    tensors = {p.name: torch.randn(p.shape, generator=torch.Generator().manual_seed(i)) for i, p in enumerate(part.parameters())}
    part.load(tensors)
    order = list(range(0, rot_dim, 2)) + list(range(1, rot_dim, 2))
    q, down = part.w_in[part.columns["q"]], part.w_in[part.columns["down"]]
    size = D + rot_dim
    for h in range(H):
        head = tensors["l0.mix.q"][h * size:(h + 1) * size]
        assert torch.equal(q[h * size:h * size + D], head[:D]) and torch.equal(q[h * size + D:(h + 1) * size], head[D:][order])
    assert torch.equal(down[:K], tensors["l0.mix.dkv"][:K]) and torch.equal(down[K:], tensors["l0.mix.dkv"][K:][order])


@pytest.mark.parametrize("rot", [(8, 500.0, STRETCHED), (64, 20000.0, STRETCHED), (24, 10000.0, (2.0, 0.5, 8.0, 100)), (6, 100.0, (3.0, 1.0, 2.0, 30)),
                                 (10, 1000.0, None)])
def test_rotation_tables(rot):
    """The package's tables against the plain frequencies; the stretched ones have pairs of every sort."""
    from models_b200.config.specs import RopeScalingSpec, RopeSpec
    from models_b200.parts import Runtime, build_part

    dims, base, s = rot
    scaling = None if s is None else RopeScalingSpec("llama3", s[0], low_freq_factor=s[1], high_freq_factor=s[2], original_max_position=s[3])
    part = build_part("position", RopeSpec(dims, base, "half", scaling), Runtime(torch.device("cpu"), "float32", max_positions=300))
    f = pr.turns({"dims": dims, "base": base, "scaling": None if s is None else dict(zip(("factor", "low", "high", "original"), s))})
    angle = torch.arange(300).double()[:, None] * f[None, :]
    assert (part.cos.double() - torch.cos(angle)).abs().max() < 1e-4 and (part.sin.double() - torch.sin(angle)).abs().max() < 1e-4
    if s is not None and dims >= 8:
        ratio = f / pr.turns({"dims": dims, "base": base})
        assert ratio[0] == 1.0 and abs(float(ratio[-1]) - 1.0 / s[0]) < 1e-12
        assert s is not STRETCHED or dims < 64 or bool(((ratio < 0.999) & (ratio > 1.001 / s[0])).any())


def test_random_weights_put_layer_norms_around_zero():
    """A weight stored as its distance from one is drawn around zero, a plain one around one."""
    from models_b200.config import config_from_dict
    from models_b200.engine.model import parameter_requests
    from models_b200.weights.random_init import random_tensors

    t = random_tensors(parameter_requests(config_from_dict(RLX["C"]).model_spec()), 5, gain_std=0.1)
    for name in ("l0.norm1", "l3.norm1", "final.norm"):
        assert abs(float(t[name].float().mean())) < 0.05 and 0.05 < float(t[name].float().std()) < 0.15
    for name in ("l1.mix.q.norm", "l1.mix.k.norm", "l0.mix.dkv.norm"):
        assert abs(float(t[name].float().mean()) - 1.0) < 0.05


# ----------------------------------------------------------------------------------- the plain implementation

def test_plain_mechanisms_by_hand():
    x = torch.tensor([[3.0, 4.0]], dtype=F)
    r = math.sqrt(12.5 + 1e-3)
    assert torch.allclose(pr.norm_around_one(x, {"n": torch.tensor([0.5, -1.0])}, "n", 1e-3), torch.tensor([[4.5 / r, 0.0]], dtype=F))
    y = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 9.0]]] * 2, dtype=F)
    rot = {"dims": 4, "base": 100.0}
    c0, s0, c1, s1 = math.cos(1), math.sin(1), math.cos(0.1), math.sin(0.1)
    assert torch.allclose(pr.rotate_half(y, rot)[1, 0], torch.tensor([c0 - 3 * s0, 2 * c1 - 4 * s1, 3 * c0 + s0, 4 * c1 + 2 * s1, 9], dtype=F))
    assert torch.allclose(pr.rotate_neighbours(y, rot)[1, 0], torch.tensor([c0 - 2 * s0, 2 * c0 + s0, 3 * c1 - 4 * s1, 4 * c1 + 3 * s1, 9], dtype=F))
    assert torch.equal(pr.rotate_half(y, rot)[0], y[0])
    assert pr.window_visible(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    one = torch.ones(1, 1, dtype=F)
    ff = lambda g, u: float(pr.clamped_feed_forward(one, {"gate": one * g, "up": one * u, "down": one}, "", {"limit": 2.0}))  # noqa: E731
    swish = lambda g: g / (1 + math.exp(-1.702 * g))  # noqa: E731
    for g, u, want in ((1, 1, swish(1) * 2), (5, 1, swish(2) * 2), (-5, 1, swish(-5) * 2), (1, 7, swish(1) * 3), (1, -7, -swish(1))):
        assert ff(g, u) == pytest.approx(want, abs=1e-12)
    x, x0 = torch.tensor([[1.0, 2.0]], dtype=F), torch.tensor([[10.0, 20.0]], dtype=F)
    w = torch.tensor([[1.0, 0.0, 0.0, 1.0], [0.0, 1.0, 2.0, 0.0]])
    assert torch.equal(pr.join(x, x0, {"loop.in": w}), torch.tensor([[21.0, 22.0]], dtype=F))


def test_plain_attention_with_one_visible_key_returns_the_projected_key():
    """A window of one: the result is Wo times the key as projected, whatever norm and rotation do."""
    g = torch.Generator().manual_seed(1)
    c = attention(4, 2, 6, 0.5, 1, (4, 10.0, None), 0)["mixer"]
    w = {"q": torch.randn(24, 9, generator=g), "k": torch.randn(12, 9, generator=g), "q.norm": torch.randn(24, generator=g),
         "k.norm": torch.randn(12, generator=g), "o": torch.randn(9, 24, generator=g)}
    h = torch.randn(5, 9, generator=g).double()
    k = (h @ w["k"].double().T).view(5, 2, 6).repeat_interleave(2, dim=1).reshape(5, 24)
    assert torch.allclose(pr.attention(h, w, "", c, 1e-5), k @ w["o"].double().T)


@pytest.mark.parametrize("name", sorted(RLX))
def test_plain_prefix_gives_prefix(name, tmp_path):
    folder = make_folder(RLX[name], 3, tmp_path)
    tokens = random_tokens(RLX[name]["vocab"], 40, 5)
    whole = plain_logits(folder, tokens)
    assert torch.allclose(plain_logits(folder, tokens[:17]), whole[:17], atol=1e-10)


def _mistakes():
    half = lambda x, rot: pr_rotate_half(x, rot)  # noqa: E731
    pr_rotate_half, pr_rotate_neighbours, plain_visible, plain_turns = pr.rotate_half, pr.rotate_neighbours, pr.window_visible, pr.turns
    return {
        "window one longer": ("window_visible", lambda T, n: plain_visible(T, n + 1 if n else n)),
        "window one shorter": ("window_visible", lambda T, n: plain_visible(T, n - 1 if n and n > 1 else n)),
        "first position unseen": ("window_visible", lambda T, n: plain_visible(T, n) & ((torch.arange(T) > 0) | (torch.arange(T)[:, None] < 1))),
        "neighbours rotated as halves": ("rotate_neighbours", half),
        "halves rotated as neighbours": ("rotate_half", lambda x, rot: pr_rotate_neighbours(x, rot)),
        "frequencies not stretched": ("turns", lambda rot: plain_turns({"dims": rot["dims"], "base": rot["base"]})),
        "norm weight without the one": ("norm_around_one", lambda x, w, name, eps: pr.over_rms(x, eps) * pr.f64(w[name])),
        "join turned round": ("join", lambda x, x0, w: torch.cat([x0, x], -1) @ pr.f64(w["loop.in"]).T),
        "join once": ("run_order", lambda config, order=pr.run_order: [(i, j and n == next(m for m, e in enumerate(order(config)) if e[1]))
                                                                       for n, (i, j) in enumerate(order(config))]),
    }


@pytest.mark.parametrize("mistake", sorted(_mistakes()))
def test_the_models_show_mistakes(mistake, tmp_path, monkeypatch):
    """A mistake planted in the plain implementation moves some model's logits by far more than the tests allow."""
    tokens = {name: random_tokens(raw["vocab"], 110, 9) for name, raw in RLX.items()}
    folders = {name: make_folder(raw, 71 + i, tmp_path) for i, (name, raw) in enumerate(RLX.items())}
    right = {name: plain_logits(folders[name], tokens[name]) for name in RLX}
    monkeypatch.setattr(pr, *_mistakes()[mistake])
    shown = [scaled_error(plain_logits(folders[name], tokens[name]), right[name]) for name in RLX]
    assert max(shown) > 5 * TOLERANCE["bfloat16"], shown
