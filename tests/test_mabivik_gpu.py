"""The Mabivik decoder in the engine against the plain implementation (tests/plain/plain_mabivik.py): each mechanism alone with
inputs made so that one key, a window's edge, a carried state or one expert decides the result, whole prompts, prompts cut into
portions, token-by-token decoding across cache pages, windows and chunks, unequal batches, slots, pages and states used again, long
decoding from CUDA graphs, and greedy generation through the public entry point."""

import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from plain import plain_mabivik as pm
from tiny import TOLERANCE, random_tokens, scaled_error
from tiny_mabivik import MBV, ROT_A, ROT_B, ROT_C, delta, latent, make_folder, mamba2, model, moe, plain_logits

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F = torch.float64


def _engine(folder, dtype, max_tokens=2048, **more):
    from models_b200.engine.loading import engine_from_folder

    return engine_from_folder(folder, dtype, max_tokens, **more)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("mabivik")
    return {name: make_folder(raw, seed=71 + i, root=root) for i, (name, raw) in enumerate(MBV.items())}


def _close(got, want, dtype):
    """Every position within three times the common bound, all but one in twenty within the bound itself, the median within half
    of it (layers pass through norms over a head or a row whose result may be small against its spread: single positions differ)."""
    got, want = torch.as_tensor(got, dtype=F).cpu(), torch.as_tensor(want, dtype=F).cpu()
    if got.dim() == 1:
        got, want = got[None], want[None]
    assert got.shape == want.shape, (got.shape, want.shape)
    errors = (got - want).abs().amax(-1) / want.abs().max().clamp_min(1e-30)
    bound = TOLERANCE[dtype]
    ok = bool((errors < 3 * bound).all()) and int((errors >= bound).sum()) <= max(1, errors.numel() // 20) \
        and (errors.numel() < 5 or float(errors.median()) < bound / 2)
    if not ok:
        print("positions", errors.numel(), "median", float(errors.median()), "largest",
              [(int(i), round(float(errors[i]), 6)) for i in errors.argsort(descending=True)[:12]])
    return ok


def _rounded(t, dtype):
    return t.to(dtype).to(F)


def _weights(shapes, seed, scale=0.2, **special):
    """Random bfloat16-exact float32 tensors; `special` names a function of (shape, generator) for some endings."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes.items():
        make = next((f for end, f in special.items() if name.endswith("." + end)), None)
        t = make(shape, g) if make else torch.randn(shape, generator=g) * scale
        out[name] = t.to(torch.bfloat16).float()
    return out


def _part(sort, spec, weights, dtype, device, max_positions=4096):
    from models_b200.parts import Runtime, build_part

    part = build_part(sort, spec, Runtime(device, dtype, max_positions=max_positions))
    part.load({n: t.to(TORCH[dtype]) if t.is_floating_point() else t for n, t in weights.items()})
    return part


def _shapes(part_spec, sort="mixer"):
    from models_b200.parts import Runtime, build_part

    return {p.name: p.shape for p in build_part(sort, part_spec, Runtime(torch.device("meta"), "float32", max_positions=1)).parameters()}


def _spec_of(layer, vocab=50, width=48, eps=1e-5):
    """The specs a configuration makes of one layer."""
    from models_b200.config import config_from_dict

    return config_from_dict(model(vocab, width, eps, 1.0, 1.0, 8, [layer])).model_spec().layers[0]


def _state_batch(counts, slots, device, starts=None):
    """What the recurrent parts read of a step."""
    cu = [0]
    for n in counts:
        cu.append(cu[-1] + n)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=device)  # noqa: E731
    return SimpleNamespace(cu_q=i32(cu), slots=i32(slots), max_q_len=max(counts), num_sequences=len(counts))


# ----------------------------------------------------------------------------------- mechanisms alone: norms, side input, experts

@pytest.mark.parametrize("width,rows", [(50, 3), (256, 70), (64, 1), (2048, 5), (33, 9), (6000, 2)])
def test_norms_on_a_result_and_the_next_readers_rows(cuda_device, width, rows):
    """x += N(y) and x += y / rms(y) w, followed by nothing, the new rows, or the new rows through another dynamic tanh; with
    arguments on both sides of the tanh's bend."""
    from models_b200.kernels import ops

    g = torch.Generator().manual_seed(width + rows)
    rnd = lambda *shape: torch.randn(*shape, generator=g)  # noqa: E731
    dev = lambda t: t.to(cuda_device).contiguous()  # noqa: E731
    x, y = rnd(rows, width), rnd(rows, width) * 2
    w, b, w2, b2 = 1 + 0.2 * rnd(width), rnd(width), 1 + 0.2 * rnd(width), rnd(width)
    norm = lambda v, alpha, ww, bb: torch.tanh(alpha * v) * ww.double() + bb.double()  # noqa: E731
    got = ops.dynamic_tanh(dev(x), 0.7, dev(w), dev(b), torch.float32)
    assert scaled_error(got.cpu(), norm(x.double(), 0.7, w, b)) < 1e-6
    pick = torch.tensor([rows - 1, 0], dtype=torch.int32, device=cuda_device)
    assert torch.equal(ops.dynamic_tanh(dev(x), 0.7, dev(w), dev(b), torch.float32, rows=pick), got[[rows - 1, 0]])
    tanh_sum = x.double() + norm(y.double(), 1.3, w, b)
    rms_sum = x.double() + pm.over_rms(y.double(), 1e-5) * w.double()
    for then, made in ((None, None), ("rows", lambda v: v), ((0.4, dev(w2), dev(b2)), lambda v: norm(v, 0.4, w2, b2))):
        for add, want in ((lambda t, d: ops.result_tanh_add(t, dev(y), 1.3, dev(w), dev(b), then, d), tanh_sum),
                          (lambda t, d: ops.result_rms_add(t, dev(y), dev(w), 1e-5, then, d), rms_sum)):
            for dtype, bound in ((torch.float32, 1e-6), (torch.bfloat16, 5e-3)):
                stream = dev(x.clone())
                out = add(stream, dtype)
                assert scaled_error(stream.cpu(), want) < 1e-6
                assert (out is None) == (then is None)
                if out is not None:
                    assert out.dtype == dtype and scaled_error(out.float().cpu(), made(want)) < bound


@pytest.mark.parametrize("top,placed", [(1, False), (3, False), (3, True)])
def test_sum_of_expert_results_inside_the_norm(cuda_device, top, placed):
    from models_b200.kernels import ops

    g = torch.Generator().manual_seed(top)
    rows, width = 11, 72
    x, slots = torch.randn(rows, width, generator=g), torch.randn(rows * top + (40 if placed else 0), width, generator=g)
    place = torch.randperm(slots.shape[0], generator=g)[:rows * top].to(torch.int32) if placed else None
    w, b = torch.randn(width, generator=g), torch.randn(width, generator=g)
    mine = slots[place.long()] if placed else slots
    want = x.double() + torch.tanh(0.9 * mine.double().view(rows, top, width).sum(1) / top) * w.double() + b.double()
    stream = x.clone().to(cuda_device)
    ops.result_tanh_add(stream, slots.to(cuda_device), 0.9, w.to(cuda_device), b.to(cuda_device), top=top,
                        position=place.to(cuda_device) if placed else None, entry_weight=1.0 / top)
    assert scaled_error(stream.cpu(), want) < 2e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,dim,index,layers,rows", [(64, 8, 0, 1, 3), (50, 7, 2, 3, 20), (256, 40, 1, 2, 200)])
def test_token_side_input(cuda_device, width, dim, index, layers, rows, dtype):
    """The layer's own columns of the token's own row: the table is constant but for one layer's columns of one token."""
    from models_b200.config.specs import TokenSideSpec

    spec = TokenSideSpec(width, 30, dim, index, layers, {"table": "t", "gate": "g", "proj": "p"})
    w = _weights({"t": (30, layers * dim), "g": (dim, width), "p": (width, dim)}, 3, 0.3)
    part = _part("feed_forward", spec, w, dtype, cuda_device)
    g = torch.Generator().manual_seed(rows)
    x = _rounded(torch.randn(rows, width, generator=g), TORCH[dtype])
    tokens = torch.randint(0, 30, (rows,), generator=g).to(torch.int32)
    tokens[0], tokens[-1] = 0, 29
    e = w["t"].double()[tokens.long(), index * dim:(index + 1) * dim]
    want = (pm.gelu_tanh(x @ w["g"].double().T) * e) @ w["p"].double().T
    got = part.forward_wide(x.to(TORCH[dtype]).to(cuda_device), SimpleNamespace(tokens=tokens.to(cuda_device)))
    assert got.dtype == torch.float32 and scaled_error(got.cpu(), want) < (2e-6 if dtype == "float32" else 1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,experts,top,ff,tokens", [(64, 6, 2, 40, 5), (64, 6, 2, 40, 90), (128, 4, 1, 64, 400), (50, 5, 3, 33, 70),
                                                         (48, 1, 1, 16, 3), (256, 8, 8, 32, 60)])
def test_experts_by_a_table(cuda_device, width, experts, top, ff, tokens, dtype):
    """The three forms the step's size picks; every expert's matrices have a scale of their own, so that one wrong expert shows."""
    layer = delta(1, 1, 8, 8, 2, moe(experts, top, ff))
    spec = _spec_of(layer, vocab=37, width=width).feed_forward
    g = torch.Generator().manual_seed(experts + tokens)
    w = {}
    for name, shape in _shapes(spec, "feed_forward").items():
        if name.endswith("table"):
            w[name] = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(37)]).to(torch.int32)
        else:
            expert = int(name.split(".e")[1].split(".")[0])
            w[name] = (torch.randn(shape, generator=g) * 0.2 * (1 + 0.3 * expert)).to(torch.bfloat16).float()
    part = _part("feed_forward", spec, w, dtype, cuda_device)
    x = _rounded(torch.randn(tokens, width, generator=g), TORCH[dtype])
    ids = torch.randint(0, 37, (tokens,), generator=g).to(torch.int32)
    want = pm.table_experts(x, w, "l0.mlp.", layer["mlp"], ids.tolist())
    batch = SimpleNamespace(tokens=ids.to(cuda_device))
    rows = x.to(TORCH[dtype]).to(cuda_device)
    got = part.forward_wide(rows, batch).double().cpu()
    bound = 5e-6 if dtype == "float32" else 1.5e-2
    assert scaled_error(got, want) < bound
    r = part.forward_results(rows, batch)
    place = r.position.long() if r.position is not None else torch.arange(tokens * top, device=cuda_device)
    assert scaled_error((r.rows[place].view(tokens, top, width).sum(1) * r.weight).cpu(), want) < bound


# ----------------------------------------------------------------------------------- mechanisms alone: attention

def _pool(T, D, page_size, device, dtype, shuffle_seed=0):
    """A fresh pool (full of NaN) with the sequence's pages in a shuffled order: pool, page table, slot mapping, positions."""
    pages = -(-T // page_size)
    order = torch.randperm(pages, generator=torch.Generator().manual_seed(shuffle_seed)) + 1
    pool = torch.full((pages + 1, 1, page_size, D), float("nan"), dtype=dtype, device=device)
    positions = torch.arange(T, dtype=torch.int32)
    mapping = (order[positions // page_size].to(torch.int32) * page_size + positions % page_size).to(torch.int32).to(device)
    return pool, order.to(torch.int32)[None, :].contiguous().to(device), mapping, positions.to(device)


def _plain_attend(q, rows, value_dim, scale, window):
    """q [T, H, D], rows [T, D] read as key and (their first value_dim numbers) as value, float64 -> [T, H, value_dim]."""
    seen = pm.window_visible(q.shape[0], window)
    out = torch.zeros(q.shape[0], q.shape[1], value_dim, dtype=F)
    for h in range(q.shape[1]):
        s = (q[:, h] @ rows.T * scale).masked_fill(~seen, float("-inf"))
        out[:, h] = torch.softmax(s, -1) @ rows[:, :value_dim]
    return out


FORMS = [("float32", "rows", 64), ("float32", "decode", 64), ("bfloat16", "rows", 64), ("bfloat16", "tc", 64), ("bfloat16", "decode", 64),
         ("float32", "decode", 32), ("bfloat16", "tc_decode", 64)]


@pytest.mark.parametrize("dtype,kernel,page_size", FORMS)
@pytest.mark.parametrize("T,window,loud", [(150, 64, 149 - 63), (150, 64, 149 - 64), (200, 72, 128), (200, 72, 127), (200, 71, 128), (130, 1, 129),
                                           (130, 1, 128), (700, 300, 401), (700, 300, 400), (700, None, 3), (65, 65, 0), (65, 64, 0), (700, 65, 650),
                                           (640, 640, 0), (641, 640, 0)])
def test_one_loud_key_at_the_windows_edge(cuda_device, dtype, kernel, page_size, T, window, loud):
    """One key stands out for the last query: seen when it lies just inside the window, without any effect just outside; rows a
    query does not see may hold anything (NaN) when the whole page before the window does."""
    from models_b200.kernels import ops

    H, D, Dv = 19 if kernel == "tc_decode" else 3, 48, 32
    td = TORCH[dtype]
    g = torch.Generator().manual_seed(T + (window or 0))
    q, rows = torch.randn(T, H, D, generator=g) * 0.3, torch.randn(T, D, generator=g) * 0.3
    rows[loud] = torch.sign(rows[loud]) * 2.0
    q[T - 1] = rows[loud] * 1.5
    q, rows = _rounded(q, td), _rounded(rows, td)
    pool, table, mapping, _ = _pool(T, D, page_size, cuda_device, td)
    pool.view(-1, D)[mapping.long()] = rows.to(td).to(cuda_device)
    q_len = 1 if "decode" in kernel else 40
    if window is not None:  # pages no query of the step sees are given back: whatever they hold must not matter
        lowest = max(0, T - q_len - window + 1)
        for block in range(lowest // page_size):
            pool[table[0, block]] = float("nan")
            table[0, block] = 0
    want = _plain_attend(q, rows, Dv, 0.5, window)[T - q_len:].reshape(q_len, -1)
    out = torch.full((q_len, H * Dv), float("nan"), dtype=td, device=cuda_device)
    i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=cuda_device)  # noqa: E731
    ops.gated_attention(q[T - q_len:].reshape(q_len, -1).to(td).to(cuda_device), out, pool, None, table, i32(0, q_len), i32(T), q_len, H, 1, D, Dv,
                        "softmax", 0.5, window=window or 0, kernel=kernel)
    assert scaled_error(out.float().cpu(), want) < (2e-6 if dtype == "float32" else 1e-2)
    inside = window is None or T - 1 - loud < window
    followed = float((want[-1].view(H, Dv) - rows[loud, :Dv]).abs().max()) < 0.5
    assert followed == inside  # the inputs do decide


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [latent(4, 16, 8, 8, 24, 32, 0.3, 9, ROT_A, None), latent(2, 64, 16, 32, 96, 112, 0.11, 70, ROT_C, None),
                                   latent(3, 10, 6, 14, 21, 26, 0.24, None, ROT_B, None), latent(1, 32, 64, 48, 40, 256, 0.1, 100, ROT_C, None)],
                         ids=["small", "tensor-cores", "odd", "wide-rows"])
def test_latent_attention_alone_whole_then_in_pieces(cuda_device, layer, dtype):
    """The part through its own kernels: a prompt whole; the same tokens as portions of 2, 60, 1 and the rest; and the decode
    form token by token, all from positions that lie across page borders."""
    spec = _spec_of(layer).mixer
    td, c = TORCH[dtype], layer["mixer"]
    w = _weights(_shapes(spec), 5, 0.25, uq=lambda s, g: torch.randn(s, generator=g) * 0.5, norm=lambda s, g: 1 + 0.2 * torch.randn(s, generator=g))
    part = _part("mixer", spec, w, dtype, cuda_device)
    T, W = 140, 48
    g = torch.Generator().manual_seed(9)
    h = _rounded(torch.randn(T, W, generator=g), td)
    want = pm.latent_attention(h, w, "l0.mix.", c, 1e-5, pm.latent_rows(h, w, "l0.mix.", c, 1e-5))
    for cuts in ([T], [2, 60, 1, 77], [70] + [1] * 70):
        pool, table, mapping, positions = _pool(T, c["kv_rank"] + c["rot_dim"], 64, cuda_device, td, len(cuts))
        at, rows = 0, []
        for n in cuts:
            batch = SimpleNamespace(positions=positions[at:at + n].contiguous(), cu_q=torch.tensor([0, n], dtype=torch.int32, device=cuda_device),
                                    kv_lens=torch.tensor([at + n], dtype=torch.int32, device=cuda_device), max_q_len=n,
                                    groups=[SimpleNamespace(block_table=table, slot_mapping=mapping[at:at + n].contiguous())])
            run = SimpleNamespace(group=0, k_pool=pool, v_pool=None, writes_cache=True)
            rows.append(part.forward(h[at:at + n].to(td).to(cuda_device), batch, run).float().cpu())
            at += n
        assert _close(torch.cat(rows), want, dtype), len(cuts)


# ----------------------------------------------------------------------------------- mechanisms alone: recurrences

SPACES = {"odd": mamba2(5, 6, 18, 5, 3, 2, None), "one": mamba2(1, 24, 8, 1, 1, 1, None), "chunks": mamba2(6, 32, 64, 3, 2, 4, None),
          "small-chunks": mamba2(4, 16, 16, 2, 4, 5, None), "large": mamba2(2, 64, 128, 1, 1, 4, None), "widest": mamba2(1, 128, 256, 1, 1, 3, None),
          "tall": mamba2(2, 8, 300, 1, 1, 2, None)}
DELTAS = {"odd": delta(6, 2, 18, 10, 3, None), "one": delta(1, 1, 8, 40, 1, None), "wide": delta(4, 4, 64, 48, 4, None)}


def _recurrent(layer, dtype, device, decays="mixed"):
    spec = _spec_of(layer).mixer
    rate = {"mixed": lambda s, g: torch.rand(s, generator=g) * 4 - 3, "lasting": lambda s, g: torch.full(s, -8.0),
            "forgetful": lambda s, g: torch.full(s, 3.0)}[decays]
    normal = lambda a, b=0.0: lambda s, g: torch.randn(s, generator=g) * a + b  # noqa: E731
    w = _weights(_shapes(spec), 21, 0.25, A_log=rate, dt_bias=normal(0.8, -0.5), conv=normal(0.6), norm=normal(0.2, 1.0), b=normal(0.3),
                 D=lambda s, g: torch.rand(s, generator=g) + 0.5)  # (near zero it could cancel dt C.B, and the norm would enlarge roundings)
    plain = pm.state_space if layer["type"] == "mamba2" else pm.gated_delta_rule
    part = _part("mixer", spec, w, dtype, device)
    return part, lambda h: plain(h, w, "l0.mix.", layer["mixer"], 1e-5)


def _state(part, slots, device):
    r = part.state_request()
    return torch.zeros((slots,) + tuple(r.shape), dtype=r.dtype, device=device)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind,name", [("space", n) for n in sorted(SPACES)] + [("delta", n) for n in sorted(DELTAS)])
def test_recurrence_ragged_carried_and_used_again(cuda_device, kind, name, dtype):
    """Unequal sequences in one step (one of a single token), continued by portions of 1, 2, 140 and 37 tokens and then token by
    token; a slot zeroed and used again starts from nothing; other slots' states are left alone."""
    layer = (SPACES if kind == "space" else DELTAS)[name]
    part, plain = _recurrent(layer, dtype, cuda_device)
    td = TORCH[dtype]
    g = torch.Generator().manual_seed(13)
    lengths = [321, 150, 1 + 1 + 2]
    hs = [_rounded(torch.randn(n, 48, generator=g), td) for n in lengths]
    want = [plain(h) for h in hs]
    state = _state(part, 5, cuda_device)
    state[3] = 7.0
    slots, at = [4, 0, 2], [0, 0, 0]
    got = [[], [], []]

    def step(counts):
        live = [i for i, n in enumerate(counts) if n]
        rows = torch.cat([hs[i][at[i]:at[i] + counts[i]] for i in live]).to(td).to(cuda_device)
        out = part.forward(rows, _state_batch([counts[i] for i in live], [slots[i] for i in live], cuda_device), SimpleNamespace(state=state)).float().cpu()
        row = 0
        for i in live:
            got[i].append(out[row:row + counts[i]])
            row += counts[i]
            at[i] += counts[i]

    for counts in ([100, 33, 1], [1, 0, 1], [2, 2, 0], [140, 37, 2], [37, 40, 0]):
        step(counts)
    for _ in range(38):
        step([1, 1, 0])
    step([3, 0, 0])
    for i in range(3):
        assert _close(torch.cat(got[i]), want[i], dtype), i
    assert bool((state[3] == 7.0).all())
    state[4].zero_()  # a slot handed out again
    at[0], got[0] = 0, []
    step([60, 0, 0])
    assert _close(got[0][0], want[0][:60], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decays", ["lasting", "forgetful"])
def test_state_space_that_keeps_and_that_forgets(cuda_device, decays, dtype):
    """Decays near one over 600 tokens (the first token still counts in the last: several chunks carry it) and near zero (large
    sums of logarithms inside a chunk)."""
    part, plain = _recurrent(SPACES["chunks"], dtype, cuda_device, decays)
    td = TORCH[dtype]
    g = torch.Generator().manual_seed(3)
    h = torch.randn(600, 48, generator=g) * 0.3
    h[0] *= 10.0  # a loud first token
    h = _rounded(h, td)
    for count in (600, 129):
        state = _state(part, 1, cuda_device)
        got = part.forward(h[:count].to(td).to(cuda_device), _state_batch([count], [0], cuda_device), SimpleNamespace(state=state))
        assert scaled_error(got.float().cpu(), plain(h[:count])) < (2e-5 if dtype == "float32" else 3e-2)


def test_chunks_and_walk_leave_the_same_state(cuda_device):
    """bfloat16: a prompt through the chunks leaves the state that walking its tokens leaves, up to the convolved rows' rounding."""
    from models_b200.kernels import ops

    part, _ = _recurrent(SPACES["large"], "bfloat16", cuda_device)
    h = torch.randn(300, 48, generator=torch.Generator().manual_seed(8)).to(torch.bfloat16).to(cuda_device)
    states = []
    for least in (32, 1000):
        before, ops.SPACE_CHUNK_MIN_ROWS = ops.SPACE_CHUNK_MIN_ROWS, least
        try:
            state = _state(part, 1, cuda_device)
            part.forward(h, _state_batch([300], [0], cuda_device), SimpleNamespace(state=state))
        finally:
            ops.SPACE_CHUNK_MIN_ROWS = before
        states.append(state.double().cpu())
    floats = part.state_floats
    assert scaled_error(states[0][:, :floats], states[1][:, :floats]) < 5e-3
    assert torch.equal(states[0][:, floats:], states[1][:, floats:])  # the convolution's stored inputs


# ----------------------------------------------------------------------------------- whole models

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MBV))
def test_whole_prompt_every_position(cuda_device, folders, name, dtype):
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], dtype)
    for n, seed in ((1, 1), (2, 5), (7, 2), (70, 3), (200, 4)):
        tokens = random_tokens(MBV[name]["vocab"], n, seed)
        slot = engine.open_slot()
        logits = engine.step([StepEntry(slot, tokens, list(range(n)))])
        engine.release_slot(slot)
        assert _close(logits, plain_logits(folders[name], tokens), dtype), (name, dtype, n)
    engine.cache.check()


@pytest.mark.parametrize("name", sorted(MBV))
def test_residual_stream_after_every_layer(cuda_device, folders, name):
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], "float32")
    tokens = random_tokens(MBV[name]["vocab"], 90, 6)
    seen = []
    engine.model.observer = lambda run, x: seen.append(x.double().cpu())
    slot = engine.open_slot()
    engine.step([StepEntry(slot, tokens, [89])])
    expected = []
    plain_logits(folders[name], tokens, expected)
    assert len(seen) == len(expected) == len(MBV[name]["layers"])
    for run, (got, want) in enumerate(zip(seen, expected)):
        assert scaled_error(got, want) < 2e-5, run


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MBV))
def test_prompt_then_token_by_token(cuda_device, folders, name, dtype):
    """A short prompt, then 130 tokens one by one: the decode form of the attention crosses cache pages and windows (pages behind
    the widest window are given back), and the recurrences with their convolutions are carried through every step."""
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], dtype)
    n, head = 150, 20
    tokens = random_tokens(MBV[name]["vocab"], n, 7)
    expected = plain_logits(folders[name], tokens)
    slot = engine.open_slot()
    rows = [engine.step([StepEntry(slot, tokens[:head], [head - 1])])]
    for i in range(head, n):
        rows.append(engine.step([StepEntry(slot, [tokens[i]], [0])]))
    assert _close(torch.cat(rows), expected[head - 1:], dtype)
    engine.cache.check()
    engine.release_slot(slot)
    assert all(g.pages.held == 0 for g in engine.cache.groups)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "D"])
def test_token_by_token_from_the_first_token(cuda_device, folders, name, dtype):
    """No prompt step at all: the first tokens of a sequence go through the decode kernels."""
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], dtype)
    tokens = random_tokens(MBV[name]["vocab"], 70, 17)
    expected = plain_logits(folders[name], tokens)
    slot = engine.open_slot()
    rows = [engine.step([StepEntry(slot, [t], [0])]) for t in tokens]
    assert _close(torch.cat(rows), expected, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,portions", [("A", [2, 3, 17, 64, 1, 2, 90, 21]), ("B", [64, 64, 2, 70]), ("C", [130, 2, 68, 200]), ("D", [5, 2, 2, 129, 62])])
def test_prompt_in_portions(cuda_device, folders, name, portions, dtype):
    """A portion starts inside a sequence: its recurrences go on from the stored states, its convolutions from the stored inputs
    (also when the portion is shorter than the convolution), its queries see the window's earlier rows."""
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], dtype)
    tokens = random_tokens(MBV[name]["vocab"], sum(portions), 8)
    expected = plain_logits(folders[name], tokens)
    slot = engine.open_slot()
    at, rows = 0, []
    for count in portions:
        rows.append(engine.step([StepEntry(slot, tokens[at:at + count], list(range(count)))]).clone())
        at += count
    assert _close(torch.cat(rows), expected, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MBV))
def test_unequal_batches_and_slots_used_again(cuda_device, folders, name, dtype):
    """Four prompts of unequal lengths in one step, decoded together while the shorter ones end; then new requests take the freed
    slots and pages (their states must start at zero, their pages hold old rows)."""
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], dtype, max_tokens=1024)
    vocab = MBV[name]["vocab"]
    for round_index in range(2):
        lengths, prompts = [1, 33, 140, 70], [1, 20, 131, 66]
        full = [random_tokens(vocab, n + 12, 10 * round_index + i) for i, n in enumerate(lengths)]
        expected = [plain_logits(folders[name], t) for t in full]
        slots = [engine.open_slot() for _ in full]
        out = engine.step([StepEntry(s, t[:p], [0, p - 1]) for s, t, p in zip(slots, full, prompts)])
        got_rows = list(out)
        want_rows = [expected[i][r] for i, p in enumerate(prompts) for r in (0, p - 1)]
        live, at = list(range(4)), list(prompts)
        while live:
            out = engine.step([StepEntry(slots[i], [full[i][at[i]]], [0]) for i in live])
            for row, i in enumerate(live):
                got_rows.append(out[row].clone())
                want_rows.append(expected[i][at[i]])
                at[i] += 1
            for i in [i for i in live if at[i] == len(full[i])]:
                engine.release_slot(slots[i])
                live.remove(i)
        assert _close(torch.stack(got_rows), torch.stack(want_rows), dtype), round_index
        engine.cache.check()
    assert engine.cache.slots.held == 0 and all(g.pages.held == 0 for g in engine.cache.groups)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_from_graphs(cuda_device, folders, name, dtype):
    """Three sequences decoded for 330 steps from captured steps, over several pages and many windows; one sequence ends on the way
    and another takes its slot (and must not inherit its states or its rows)."""
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], dtype, max_tokens=4096)
    engine.enable_decode_graphs(4)
    vocab = MBV[name]["vocab"]
    full = [random_tokens(vocab, n, 20 + i) for i, n in enumerate((340, 200, 150, 120))]
    expected = [plain_logits(folders[name], t) for t in full]
    prompts = [5, 70, 1, 30]
    slots = {i: engine.open_slot() for i in range(3)}
    engine.step([StepEntry(slots[i], full[i][:prompts[i]], []) for i in range(3)])
    at = {i: prompts[i] for i in range(3)}
    got_rows, want_rows = [], []
    while at:
        live = sorted(at)
        out = engine.decode([slots[i] for i in live], [full[i][at[i]] for i in live])
        for row, i in enumerate(live):
            if at[i] % 7 == 0 or at[i] > len(full[i]) - 3:
                got_rows.append(out[row].clone())
                want_rows.append(expected[i][at[i]])
            at[i] += 1
            if at[i] == len(full[i]):
                engine.release_slot(slots.pop(i))
                del at[i]
                if i == 2:  # a new request in the freed slot, from its prompt
                    slots[3] = engine.open_slot()
                    engine.step([StepEntry(slots[3], full[3][:prompts[3]], [])])
                    at[3] = prompts[3]
    assert _close(torch.stack(got_rows), torch.stack(want_rows), dtype)
    assert engine.decode_graphs.captured  # the steps did come from captures
    engine.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["recurrent", "attention"])
def test_models_of_one_kind_of_layer(cuda_device, tmp_path, kind, dtype):
    """Only recurrent layers (no cache group at all) or only attentions (no state: short prompt steps may come from captures too),
    the latter with a reader that sees farther than the rows' owner: prompts of one length class four times over, then tokens
    one by one from captured decode steps."""
    from models_b200.engine import StepEntry

    layers = {"recurrent": [mamba2(4, 16, 16, 2, 1, 4, moe(4, 2, 24)), delta(2, 2, 16, 16, 3, None)],
              "attention": [latent(4, 16, 16, 8, 24, 32, 0.25, 10, ROT_B, moe(4, 2, 24)), latent(2, 16, 16, 16, 16, 32, 0.3, 90, ROT_B, None, kv_from=0)]}[kind]
    raw = model(120, 64, 1e-5, 1.0, 0.5, 8, layers)
    folder = make_folder(raw, 90, tmp_path)
    engine = _engine(folder, dtype, 1024)
    engine.enable_decode_graphs(4)
    assert (len(engine.cache.groups) == 0) == (kind == "recurrent") and (not engine.state.tensors) == (kind == "attention")
    for seed in range(4):
        tokens = random_tokens(120, 140, seed)
        want = plain_logits(folder, tokens)
        slot = engine.open_slot()
        rows = [engine.step([StepEntry(slot, tokens[:100], [99])])]
        for t in tokens[100:]:
            rows.append(engine.decode([slot], [t]).clone())
        assert _close(torch.cat(rows), want[99:], dtype), seed
        engine.release_slot(slot)
    engine.cache.check()


MBV_MID = model(1000, 384, 1e-6, 0.8, 0.6, 36, [
    latent(6, 48, 24, 80, 120, 168, 0.11, 96, (30000.0, (3.0, 400.0, 24.0, 1.5)), moe(24, 5, 96)),
    mamba2(9, 80, 80, 3, 9, 3, moe(10, 2, 128)),
    delta(6, 3, 48, 80, 3, moe(6, 1, 200)),
    latent(5, 40, 24, 24, 72, 168, 0.13, 250, (30000.0, (3.0, 400.0, 24.0, 1.5)), moe(7, 3, 64), kv_from=0),
])


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_mid_sized_model_long_prompts_and_batches(cuda_device, tmp_path, dtype):
    """Sizes between the small configurations and the benchmark's: a prompt of 700 tokens whole, then decoded across window edges;
    three unequal prompts in one step (1, 300 and 650 tokens), then decoded together while the short one ends."""
    from models_b200.engine import StepEntry

    folder = make_folder(MBV_MID, 77, tmp_path)
    engine = _engine(folder, dtype, max_tokens=4096)
    vocab = MBV_MID["vocab"]
    tokens = random_tokens(vocab, 740, 5)
    expected = plain_logits(folder, tokens)
    want_rows = [0, 95, 96, 97, 127, 128, 249, 250, 251, 383, 384, 500, 699]
    slot = engine.open_slot()
    rows = [engine.step([StepEntry(slot, tokens[:700], want_rows)])]
    for i in range(700, 740):
        rows.append(engine.step([StepEntry(slot, [tokens[i]], [0])]))
    assert _close(torch.cat(rows), torch.cat([expected[want_rows], expected[700:]]), dtype)
    engine.release_slot(slot)
    lengths, prompts = [9, 330, 680], [1, 300, 650]
    full = [random_tokens(vocab, n, 30 + i) for i, n in enumerate(lengths)]
    wanted = [plain_logits(folder, t) for t in full]
    slots = [engine.open_slot() for _ in full]
    out = engine.step([StepEntry(s, t[:p], [p - 1]) for s, t, p in zip(slots, full, prompts)])
    got, want = [out], [torch.stack([wanted[i][p - 1] for i, p in enumerate(prompts)])]
    live, at = [0, 1, 2], list(prompts)
    while live:
        out = engine.step([StepEntry(slots[i], [full[i][at[i]]], [0]) for i in live])
        got.append(out.clone())
        want.append(torch.stack([wanted[i][at[i]] for i in live]))
        for i in list(live):
            at[i] += 1
            if at[i] == len(full[i]):
                engine.release_slot(slots[i])
                live.remove(i)
    assert _close(torch.cat(got), torch.cat(want), dtype)
    engine.cache.check()


def test_logits_do_not_depend_on_the_batch_or_the_cut(cuda_device, folders):
    """float32: the same position through a whole prompt, through portions, and inside a batch differs by rounding only."""
    from models_b200.engine import StepEntry

    for name in ("A", "C"):
        engine = _engine(folders[name], "float32")
        vocab = MBV[name]["vocab"]
        a, b = random_tokens(vocab, 100, 31), random_tokens(vocab, 37, 32)
        slot = engine.open_slot()
        whole = engine.step([StepEntry(slot, a, [99])])
        engine.release_slot(slot)
        s1, s2 = engine.open_slot(), engine.open_slot()
        engine.step([StepEntry(s2, b[:30], []), StepEntry(s1, a[:64], [])])
        engine.step([StepEntry(s1, a[64:99], []), StepEntry(s2, b[30:], [])])
        cut = engine.step([StepEntry(s1, a[99:], [0])])
        assert scaled_error(cut, whole) < 5e-6, name


def test_greedy_generation_through_the_entry_point(cuda_device, folders):
    import models_b200

    folder = folders["A"]
    prompts = [random_tokens(MBV["A"]["vocab"], n, 50 + n) for n in (3, 40, 11)]
    steps = 40
    config, weights = pm.read_model_folder(folder)
    expected, margins = [], []
    for prompt in prompts:
        tokens, out, margin = list(prompt), [], []
        for _ in range(steps):
            logits = pm.forward(config, weights, tokens)[-1]
            top = torch.topk(logits, 2).values
            margin.append(float(top[0] - top[1]))
            out.append(int(torch.argmax(logits)))
            tokens.append(out[-1])
        expected.append(out)
        margins.append(margin)
    for dtype in DTYPES:
        generator = models_b200.load_model(folder, dtype=dtype, max_batch=4, context=256)
        results = generator.generate_batch(prompts, models_b200.SamplingOptions(temperature=0.0, max_tokens=steps))
        for result, want, margin in zip(results, expected, margins):
            for i, (a, b) in enumerate(zip(result.tokens, want)):
                if a != b:
                    assert dtype == "bfloat16" and margin[i] < 0.05, (dtype, i, result.tokens, want)
                    break
        generator.close()


def test_trace_replay_program(cuda_device, folders, tmp_path):
    """bin/trace_run on a Mabivik folder: two prompts in one step, then decoded together from captured steps."""
    name = "D"
    vocab = MBV[name]["vocab"]
    a, b = random_tokens(vocab, 90, 1), random_tokens(vocab, 12, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:70], "want": [0, 69]}, {"id": "b", "tokens": b[:5], "want": [4]}], "end": []}]
    for i in range(20):
        entries = [{"id": "a", "tokens": [a[70 + i]], "want": [0]}]
        if i < 7:
            entries.append({"id": "b", "tokens": [b[5 + i]], "want": [0]})
        steps.append({"step": i + 1, "entries": entries, "end": (["b"] if i == 6 else []) + (["a"] if i == 19 else [])})
    out = tmp_path / "out"
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    ea, eb = plain_logits(folders[name], a), plain_logits(folders[name], b)
    for dtype in DTYPES:
        proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(folders[name]), "--dtype", dtype,
                               "--out", str(out), "--max-tokens", "102"],
                              input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900)
        assert proc.returncode == 0, proc.stderr[-2000:]
        first = np.fromfile(out / "0.f32", dtype="<f4").reshape(3, vocab)
        got, want = [first[0], first[1], first[2]], [ea[0], ea[69], eb[4]]
        for i in range(20):
            rows = np.fromfile(out / f"{i + 1}.f32", dtype="<f4").reshape(-1, vocab)
            got.append(rows[0])
            want.append(ea[70 + i])
            if i < 7:
                got.append(rows[1])
                want.append(eb[5 + i])
        assert _close(np.stack(got), torch.stack(want), dtype), dtype
