"""Mabivik without a GPU: the configuration reader (round trip, refusals, the tensors a model asks for), the cache bookkeeping of
layers that read other layers' rows, expert tables, and the plain implementation against cases worked out by hand and against
itself (a prefix of a sequence gives the prefix of its logits)."""

import copy
import math

import pytest
import torch

from plain import plain_mabivik as pm
from tiny import random_tokens
from tiny_mabivik import MBV, ROT_A, delta, latent, make_folder, mamba2, model, moe

F = torch.float64


@pytest.mark.parametrize("name", sorted(MBV))
def test_configuration_round_trip_and_tensors(name):
    from models_b200.config import config_from_dict
    from models_b200.engine.model import parameter_requests

    raw = MBV[name]
    config = config_from_dict(raw)
    assert config.to_dict() == raw
    spec = config.model_spec()
    assert not spec.head.tied and spec.head.logit_scale == raw["logit_scale"] and spec.embedding.scale == raw["embedding"]["scale"]
    W, side, count = raw["width"], raw["token_side"]["dim"], len(raw["layers"])
    requests = parameter_requests(spec)
    assert requests["head"].shape == (raw["vocab"], W) and requests["side.embed"].shape == (raw["vocab"], side * count)
    assert requests["final.norm.alpha"].shape == () and requests["final.norm.b"].shape == (W,)
    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for norm in ("norm1", "norm1b"):
            assert requests[p + norm].shape == requests[p + norm + ".b"].shape == (W,) and requests[p + norm + ".alpha"].shape == ()
        assert ((p + "norm2") in requests) == ((p + "norm2b.alpha") in requests) == (layer["mlp"] is not None)
        assert requests[p + "side.gate"].shape == (side, W) and requests[p + "side.proj"].shape == (W, side)
        assert spec.schedule[i].cache_from == m.get("kv_from")
        if layer["type"] == "delta":
            assert requests[p + "mix.k.conv"].shape == (m["kv_heads"] * m["dim"], m["conv"]) and requests[p + "mix.norm"].shape == (m["vdim"],)
        elif layer["type"] == "latent_attention":
            assert requests[p + "mix.uq"].shape == (m["heads"] * (m["dim"] + m["rot_dim"]), m["q_rank"])
            assert requests[p + "mix.uk"].shape == (m["heads"] * m["dim"], m["kv_rank"]) and requests[p + "mix.g"].shape == (m["heads"] * m["vdim"], W)
            own = m.get("kv_from") is None
            assert ((p + "mix.dkv") in requests) == ((p + "mix.dkv.norm") in requests) == own
            if own:
                assert requests[p + "mix.dkv"].shape == (m["kv_rank"] + m["rot_dim"], W)
        else:
            inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
            assert requests[p + "mix.in"].shape == (2 * inner + 2 * gn + m["heads"], W) and requests[p + "mix.conv.b"].shape == (inner + 2 * gn,)
        if layer["mlp"]:
            r = layer["mlp"]["router"]
            assert requests[p + "mlp.table"].shape == (raw["vocab"], r["top"]) and requests[p + "mlp.table"].kind == "table"
            assert (p + f"mlp.e{r['experts'] - 1}.down") in requests and (p + f"mlp.e{r['experts']}.down") not in requests


def test_configurations_that_are_refused():
    from models_b200.config import ConfigError, config_from_dict

    good = model(50, 16, 1e-5, 1.0, 1.0, 4, [
        latent(2, 8, 4, 8, 8, 8, 0.3, 4, ROT_A, moe(3, 2, 8)), delta(2, 1, 8, 8, 2, None), mamba2(4, 4, 8, 2, 2, 2, None),
        latent(1, 8, 4, 8, 8, 8, 0.3, 9, ROT_A, None, kv_from=0)])
    config_from_dict(good)
    mixer = lambda c, i: c["layers"][i]["mixer"]  # noqa: E731
    for change in (lambda c: mixer(c, 1).update(heads=3, kv_heads=2),
                   lambda c: mixer(c, 0)["rot"].update(dims=6),            # not rot_dim
                   lambda c: mixer(c, 3).update(kv_from=1),                # a layer without latent rows
                   lambda c: mixer(c, 3).update(kv_from=3),                # itself
                   lambda c: mixer(c, 3).update(kv_rank=16),               # rows of another size
                   lambda c: mixer(c, 3)["rot"].update(base=77.0),         # another rotation
                   lambda c: mixer(c, 2).update(groups=3),
                   lambda c: mixer(c, 2).update(norm_groups=3),
                   lambda c: c["layers"][0]["mlp"]["router"].update(top=4),
                   lambda c: c["layers"][0].update(type="other"),
                   lambda c: c.pop("vocab")):
        bad = copy.deepcopy(good)
        change(bad)
        with pytest.raises(ConfigError):
            config_from_dict(bad)
    again = copy.deepcopy(good)
    again["layers"].append(latent(1, 8, 4, 8, 8, 8, 0.3, 9, ROT_A, None, kv_from=3))  # a reader of a reader
    with pytest.raises(ConfigError):
        config_from_dict(again)


def test_rows_stay_as_long_as_their_widest_reader_needs_them():
    from models_b200.cache import KvCache
    from models_b200.cache.kv_cache import KvRequest

    narrow, wide, everything = KvRequest(1, 12, 5, 0), KvRequest(1, 12, 130, 0), KvRequest(1, 12, None, 0)
    for readers, kept_from in (([narrow], 196), ([wide, narrow], 71), ([everything], 0)):
        cache = KvCache([narrow] + readers, [None] + [0] * len(readers), 64 * 10)
        assert len(cache.groups) == 1 and all(cache.run_location[i] == (0, 0) for i in range(1 + len(readers)))
        slot = cache.open_slot()
        cache.append([(slot, 200)])
        cache.commit([(slot, 200)])
        held = [p >= 0 for p in cache.groups[0].tables[slot]]
        assert held == [(b + 1) * 64 > kept_from for b in range(4)]
        cache.check()
    # readers of one layer do not widen another layer's window of the same shape
    cache = KvCache([narrow, narrow, wide], [None, None, 0], 64 * 10)
    assert [g.request.window for g in cache.groups] == [130, 5]


def test_tables_are_checked_and_drawn():
    from models_b200.config import config_from_dict
    from models_b200.engine.model import parameter_requests
    from models_b200.weights import load_tensors, random_tensors, write_random_model
    from models_b200.weights.loader import WeightsError
    from models_b200.weights.safetensors_io import write_safetensors
    import tempfile

    config = config_from_dict(model(40, 16, 1e-5, 1.0, 1.0, 4, [delta(1, 1, 8, 8, 2, moe(5, 3, 8))]))
    requests = parameter_requests(config.model_spec())
    tensors = random_tensors(requests, 7)
    table = tensors["l0.mlp.table"]
    assert table.dtype == torch.int32 and int(table.min()) >= 0 and int(table.max()) < 5 and len(table.unique()) == 5
    assert all(len(set(row)) == 3 for row in table.tolist())
    with tempfile.TemporaryDirectory() as root:
        folder = write_random_model(root, config, 7)
        assert torch.equal(load_tensors(folder, requests)["l0.mlp.table"], table)
        for change in (lambda t: t[0].fill_(2), lambda t: t[3, 0].fill_(5), lambda t: t[3, 0].fill_(-1)):
            bad = table.clone()
            change(bad)
            write_safetensors(folder / "model.safetensors", dict(tensors, **{"l0.mlp.table": bad}))
            with pytest.raises(WeightsError, match="l0.mlp.table"):
                load_tensors(folder, requests)


def test_window_counts_the_query_itself():
    assert pm.window_visible(4, 2).tolist() == [[True, False, False, False], [True, True, False, False], [False, True, True, False],
                                                [False, False, True, True]]
    assert pm.window_visible(3, 1).tolist() == torch.eye(3, dtype=torch.bool).tolist()
    assert pm.window_visible(3, None).tolist() == torch.ones(3, 3, dtype=torch.bool).tril().tolist()


def test_stretched_frequencies_by_hand():
    rot = {"dims": 8, "base": 100.0, "scaling": {"factor": 4.0, "original": 200.0, "fast": 8.0, "slow": 1.0}}
    pair = lambda t: 8 * math.log(200.0 / (2 * math.pi * t)) / (2 * math.log(100.0))  # noqa: E731
    assert (math.floor(pair(8.0)), math.ceil(pair(1.0))) == (1, 4)
    got, magnitude = pm.stretched_frequencies(rot)
    plain = [100.0 ** (-i / 4) for i in range(4)]
    ramp = [0.0, 0.0, 1 / 3, 2 / 3]
    assert got == pytest.approx([f / 4 * r + f * (1 - r) for f, r in zip(plain, ramp)])
    assert magnitude == pytest.approx(0.1 * math.log(4.0) + 1.0)
    # the product's tables are the same
    from models_b200.config import config_from_dict
    from models_b200.parts import Runtime, build_part

    raw = model(10, 16, 1e-5, 1.0, 1.0, 4, [latent(1, 8, 8, 8, 8, 8, 0.3, 4, (100.0, (4.0, 200.0, 8.0, 1.0)), None)])
    spec = config_from_dict(raw).model_spec().layers[0].mixer.position
    rope = build_part("position", spec, Runtime(torch.device("cpu"), "float32", max_positions=50))
    angle = torch.arange(50, dtype=F)[:, None] * torch.tensor(got, dtype=F)
    assert torch.allclose(rope.cos.double(), torch.cos(angle) * magnitude, atol=2e-6) and torch.allclose(rope.sin.double(), torch.sin(angle) * magnitude, atol=2e-6)


def test_state_space_by_hand():
    """One head, one state row, one column, an input matrix that hands the token through: S <- e^(-dt) S + dt B x, y = S C + D x."""
    lam = math.log(math.e - 1.0)  # softplus(lam) = 1
    w = {"m.in": torch.tensor([[50.0], [1.0], [2.0], [3.0], [0.0]], dtype=F), "m.conv": torch.ones(3, 1, dtype=F), "m.conv.b": torch.zeros(3, dtype=F),
         "m.dt_bias": torch.tensor([lam], dtype=F), "m.A_log": torch.zeros(1, dtype=F), "m.D": torch.tensor([0.5], dtype=F),
         "m.norm": torch.ones(1, dtype=F), "m.o": torch.ones(1, 1, dtype=F)}
    x = torch.tensor([[1.0], [2.0], [-1.0]], dtype=F)
    xs, bs, cs = (pm.silu(x.flatten() * f).tolist() for f in (1.0, 2.0, 3.0))
    S, want = 0.0, []
    for t in range(3):
        S = math.exp(-1.0) * S + bs[t] * xs[t]
        y = S * cs[t] + 0.5 * xs[t]
        z = 50.0 * float(x[t, 0])
        want.append(y * z / (1 + math.exp(-z)))
    c = {"heads": 1, "vdim": 1, "state": 1, "groups": 1, "norm_groups": 1, "conv": 1}
    got = pm.state_space(x, w, "m.", c, 1e18).flatten() * 1e9  # (a huge eps: the norm divides by sqrt(eps) alone)
    assert torch.allclose(got, torch.tensor(want, dtype=F), rtol=1e-5, atol=1e-12)


@pytest.mark.parametrize("name", sorted(MBV))
def test_a_prefix_gives_the_prefix_of_the_logits(tmp_path, name):
    folder = make_folder(MBV[name], 5, tmp_path)
    config, weights = pm.read_model_folder(folder)
    tokens = random_tokens(MBV[name]["vocab"], 30, 3)
    whole = pm.forward(config, weights, tokens)
    assert torch.allclose(pm.forward(config, weights, tokens[:11]), whole[:11], rtol=1e-9, atol=1e-12)
    assert bool(torch.isfinite(whole).all())
