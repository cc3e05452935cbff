"""The Rulunex decoder in the engine against the plain implementation (tests/plain/plain_rulunex.py): each mechanism alone with
inputs made so that one key, a window's edge or a bound decides the result, whole prompts, prompts cut into portions, token-by-token
decoding across cache pages and windows, unequal batches, slots and pages used again, long decoding from CUDA graphs, and greedy
generation through the public entry point."""

import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from plain import plain_rulunex as pr
from tiny import TOLERANCE, random_tokens, scaled_error
from tiny_rulunex import RLX, STRETCHED, attention, latent, make_folder, model, plain_logits

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F = torch.float64


def _engine(folder, dtype, max_tokens=2048, **more):
    from models_b200.engine.loading import engine_from_folder

    return engine_from_folder(folder, dtype, max_tokens, **more)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("rulunex")
    return {name: make_folder(raw, seed=71 + i, root=root) for i, (name, raw) in enumerate(RLX.items())}


def _close(got, want, dtype):
    """Every position within three times the common bound, all but one in twenty within the bound itself, the median within half
    of it (a looped span enlarges roundings: single positions differ)."""
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
    part.load({n: t.to(TORCH[dtype]) for n, t in weights.items()})
    return part


def _shapes(part_spec, sort="mixer"):
    from models_b200.parts import Runtime, build_part

    return {p.name: p.shape for p in build_part(sort, part_spec, Runtime(torch.device("meta"), "float32", max_positions=1)).parameters()}


def _spec_of(layer, width=48, eps=1e-5):
    """The specs a configuration makes of one layer."""
    from models_b200.config import config_from_dict

    return config_from_dict(model(50, width, eps, 1.0, None, [layer])).model_spec().layers[0]


# ----------------------------------------------------------------------------------- mechanisms alone: products, norm, feed-forward, join

def _clamped(gate, up, limit, slope, offset):
    g, u = gate.clamp(max=limit), up.clamp(min=-limit, max=limit)
    return g * torch.sigmoid(slope * g) * (u + offset)


@pytest.mark.parametrize("rows", [1, 2, 7, 8])
@pytest.mark.parametrize("plain,pairs,k", [(8, 8, 64), (24, 40, 48), (200, 96, 256), (16, 3, 1024), (2080, 1536, 512), (40, 24, 8192)])
def test_product_with_two_kinds_of_rows(cuda_device, plain, pairs, k, rows):
    """Rows stored as they are and gate/up pairs, both branches reaching past their bounds: from bfloat16 rows, from float32 rows that
    the product normalises, and from rows with parts of their sums of squares; the pairs go to a column slice whose neighbours stay."""
    from models_b200.kernels import ops

    g = torch.Generator().manual_seed(plain + pairs + k)
    dev = lambda t, d=torch.bfloat16: t.to(d).to(cuda_device).contiguous()  # noqa: E731
    w = _rounded(torch.randn(plain + 2 * pairs, k, generator=g) * k ** -0.5, torch.bfloat16)
    xf, gain = torch.randn(rows, k, generator=g) * 3, 1 + 0.3 * torch.randn(k, generator=g)
    clamp = (0.7, 1.702, 1.0)

    def check(out, wide, h):
        want = h @ w.T
        mid = _clamped(want[:, plain:plain + pairs], want[:, plain + pairs:], *clamp)
        assert scaled_error(out.double().cpu(), want[:, :plain]) < 1.5e-2
        assert scaled_error(wide[:, 8:8 + pairs].double().cpu(), mid) < 2e-2
        assert bool((wide[:, :8] == 7).all()) and bool((wide[:, 8 + pairs:] == 7).all())

    make = lambda: torch.full((rows, pairs + 24), 7.0, dtype=torch.bfloat16, device=cuda_device)  # noqa: E731
    wide, x = make(), _rounded(xf, torch.bfloat16)
    check(ops.skinny_gemm_pairs(dev(w), plain, wide[:, 8:8 + pairs], clamp, x=dev(x)), wide, x)
    wide = make()
    normed = pr.over_rms(xf.double(), 1e-4) * gain.double()
    check(ops.skinny_gemm_pairs(dev(w), plain, wide[:, 8:8 + pairs], clamp, xf=dev(xf, torch.float32), gain=dev(gain, torch.float32), eps=1e-4), wide, normed)
    parts = torch.zeros((3, ops.SSQ_COLUMNS), dtype=torch.float32, device=cuda_device)
    squares = (xf.double() ** 2).sum(1)
    parts[0, :rows], parts[2, :rows] = dev(squares * 0.25, torch.float32), dev(squares * 0.75, torch.float32)
    wide = make()
    check(ops.skinny_gemm_pairs(dev(w), plain, wide[:, 8:8 + pairs], clamp, x=dev(xf * gain), norm_parts=(parts, 3, k, 1e-4)), wide, normed)


@pytest.mark.parametrize("rows", [9, 40, 128, 129, 300])
@pytest.mark.parametrize("pairs,k", [(40, 64), (264, 520), (1024, 256)])
def test_clamped_pairs_in_the_tensor_core_products(cuda_device, rows, pairs, k):
    from models_b200.kernels import ops

    g = torch.Generator().manual_seed(rows + pairs)
    w = _rounded(torch.randn(2 * pairs, k, generator=g) * k ** -0.5, torch.bfloat16)
    x = _rounded(torch.randn(rows, k, generator=g) * 3, torch.bfloat16)
    wide = torch.full((rows, pairs + 16), 7.0, dtype=torch.bfloat16, device=cuda_device)
    both = x @ w.T
    for clamp in ((0.7, 1.702, 1.0), (2.5, 1.0, 0.0)):
        ops.tensor_core_gemm(x.to(torch.bfloat16).to(cuda_device), w.to(torch.bfloat16).to(cuda_device), ops.EPI_CLAMPED, out=wide[:, 8:8 + pairs], clamp=clamp)
        assert scaled_error(wide[:, 8:8 + pairs].double().cpu(), _clamped(both[:, :pairs], both[:, pairs:], *clamp)) < 2e-2
        assert bool((wide[:, :8] == 7).all()) and bool((wide[:, 8 + pairs:] == 7).all())
    with pytest.raises(ops.KernelError):
        ops.tensor_core_gemm(x.to(torch.bfloat16).to(cuda_device), w.to(torch.bfloat16).to(cuda_device), ops.EPI_CLAMPED)


@pytest.mark.parametrize("rows", [1, 5, 60])
def test_a_product_leaves_the_streams_rows_in_place(cuda_device, rows):
    """x += a product, with the new x also stored in the left half of a wider tensor (a gain of ones)."""
    from models_b200.kernels import ops

    g = torch.Generator().manual_seed(rows)
    n, k = 136, 96
    w, a = torch.randn(n, k, generator=g).to(torch.bfloat16), torch.randn(rows, k, generator=g).to(torch.bfloat16)
    x = torch.randn(rows, n, generator=g)
    stream, wide = x.clone().to(cuda_device), torch.full((rows, 2 * n), 7.0, dtype=torch.bfloat16, device=cuda_device)
    ones = torch.ones(n, device=cuda_device)
    more = {"out": stream, "emit_gain": ones, "emit_rows": wide[:, :n]}
    if rows <= 8:
        ops.skinny_gemm(w.to(cuda_device), ops.EPI_RESIDUAL, x=a.to(cuda_device), **more)
    else:
        ops.wide_gemm(a.to(cuda_device), w.to(cuda_device), ops.EPI_RESIDUAL, **more)
    assert scaled_error(stream.cpu(), x.double() + a.double() @ w.double().T) < 1e-5
    assert torch.equal(wide[:, :n], stream.to(torch.bfloat16)) and bool((wide[:, n:] == 7).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,rows", [(50, 3), (64, 1), (256, 200), (33, 9)])
def test_norm_with_its_weight_around_one(cuda_device, width, rows, dtype):
    from models_b200.config.specs import NormSpec

    w = _weights({"l.n": (width,)}, width, 0.4)
    part = _part("norm", NormSpec(width, 1e-3, {"weight": "l.n"}, gain_offset=1.0), w, dtype, cuda_device)
    x = torch.randn(rows, width, generator=torch.Generator().manual_seed(2))
    want = pr.norm_around_one(x.double(), w, "l.n", 1e-3)
    assert scaled_error(part.forward(x.to(cuda_device)).double().cpu(), want) < (1e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff,rows", [(48, 40, 3), (50, 33, 20), (256, 192, 200), (64, 1, 5)])
def test_clamped_feed_forward(cuda_device, width, ff, rows, dtype):
    """Gate and up values on both sides of their bounds (the gate has none below)."""
    layer = attention(1, 1, 8, 0.3, None, None, ff, 0.9)
    spec = _spec_of(layer, width).feed_forward
    w = _weights(_shapes(spec, "feed_forward"), ff, 2.0 * width ** -0.5)
    part = _part("feed_forward", spec, w, dtype, cuda_device)
    x = _rounded(torch.randn(rows, width, generator=torch.Generator().manual_seed(rows)), TORCH[dtype])
    want = pr.clamped_feed_forward(x, w, "l0.mlp.", layer["mlp"])
    gate = x @ w["l0.mlp.gate"].double().T
    assert bool((gate > 0.9).any()) and bool((gate < -0.9).any())
    assert scaled_error(part.forward(x.to(TORCH[dtype]).to(cuda_device)).double().cpu(), want) < (2e-6 if dtype == "float32" else 1.5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,rows", [(50, 3), (64, 1), (64, 8), (256, 30), (256, 200), (33, 9)])
def test_join_of_the_stream_and_the_embedding(cuda_device, width, rows, dtype):
    """At the model's start, later, and twice in a row; the embedding's rows are kept from `begin` on."""
    from models_b200.config.specs import StreamJoinSpec

    w = _weights({"loop.in": (width, 2 * width)}, width, width ** -0.5)
    part = _part("join", StreamJoinSpec(width, {"weight": "loop.in"}), w, dtype, cuda_device)
    g = torch.Generator().manual_seed(rows)
    x0, x = torch.randn(rows, width, generator=g), torch.randn(rows, width, generator=g) * 2
    bound = 2e-6 if dtype == "float32" else 1e-2
    for at_once in (True, False):
        start = x0.clone().to(cuda_device)
        part.begin(start, at_once)
        now = start if at_once else x.to(cuda_device)
        start_value = x0 if at_once else x
        first = part.forward(now, None)
        assert first.dtype == torch.float32 and scaled_error(first.cpu(), pr.join(start_value.double(), x0.double(), w)) < bound
        again = part.forward(first, None)
        assert scaled_error(again.cpu(), pr.join(first.double().cpu(), x0.double(), w)) < bound
        part.end()


# ----------------------------------------------------------------------------------- mechanisms alone: attention

def _paged(T, page_size, device, seed):
    """The sequence's pages in a shuffled order: how many, page table, slot mapping, positions."""
    pages = -(-T // page_size)
    order = torch.randperm(pages, generator=torch.Generator().manual_seed(seed)) + 1
    positions = torch.arange(T, dtype=torch.int32)
    mapping = (order[positions // page_size].to(torch.int32) * page_size + positions % page_size).to(torch.int32).to(device)
    return pages, order.to(torch.int32)[None, :].contiguous().to(device), mapping, positions.to(device)


def _run_in_pieces(part, h, cuts, dtype, device):
    """The mixer over one sequence in steps of the given sizes, through a fresh cache full of NaN; before every step the pages that no
    later query can see are given back and spoilt."""
    td, T = TORCH[dtype], h.shape[0]
    request = part.kv_request()
    pages, table, mapping, positions = _paged(T, 64, device, len(cuts))
    pool = lambda size: torch.full((pages + 1, request.num_kv_heads, 64, size), float("nan"), dtype=td, device=device)  # noqa: E731
    value_dim = request.head_dim if request.value_dim is None else request.value_dim
    k_pool, v_pool = pool(request.head_dim), pool(value_dim) if value_dim else None
    at, rows = 0, []
    for n in cuts:
        if request.window is not None:
            for block in range(max(0, at - request.window + 1) // 64):
                if int(table[0, block]):
                    for p in (k_pool, v_pool):
                        if p is not None:
                            p[table[0, block]] = float("nan")
                    table[0, block] = 0
        batch = SimpleNamespace(positions=positions[at:at + n].contiguous(), cu_q=torch.tensor([0, n], dtype=torch.int32, device=device),
                                kv_lens=torch.tensor([at + n], dtype=torch.int32, device=device), max_q_len=n,
                                fresh=at == 0, groups=[SimpleNamespace(block_table=table, slot_mapping=mapping[at:at + n].contiguous())])
        run = SimpleNamespace(group=0, k_pool=k_pool, v_pool=v_pool, writes_cache=True)
        rows.append(part.forward(h[at:at + n].to(td).to(device), batch, run).float().cpu())
        at += n
    return torch.cat(rows)


@pytest.mark.parametrize("heads,kv_heads,dim,value_dim", [(4, 2, 128, 128), (3, 1, 64, 64), (2, 2, 64, 128), (2, 1, 192, 128), (2, 2, 256, 64)])
@pytest.mark.parametrize("window", [None, 1, 64, 65, 130])
def test_prompt_attention_on_pages_unequal_and_continued(cuda_device, heads, kv_heads, dim, value_dim, window):
    """The tcgen05 form with float weights over pages full of NaN where nothing was written: a batch of prompts of unequal lengths, one
    of which goes on where earlier steps left it; loud keys that move the running maximum late."""
    from models_b200.kernels import ops

    g = torch.Generator().manual_seed(dim + (window or 0))
    lengths, counts = [300, 64, 1, 129, 200], [300, 64, 1, 129, 70]
    bf = torch.bfloat16
    pages = [-(-n // 64) for n in lengths]
    table = torch.zeros((len(lengths), max(pages)), dtype=torch.int32)
    order = (torch.randperm(sum(pages), generator=g) + 1).to(torch.int32)
    at = 0
    for i, n in enumerate(pages):
        table[i, :n] = order[at:at + n]
        at += n
    k_pool = torch.full((at + 1, kv_heads, 64, dim), float("nan"), dtype=bf, device=cuda_device)
    v_pool = torch.full((at + 1, kv_heads, 64, value_dim), float("nan"), dtype=bf, device=cuda_device)
    scale, wants, qs = 0.6 * dim ** -0.5, [], []
    for i, (n, count) in enumerate(zip(lengths, counts)):
        q, k, v = (_rounded(torch.randn(n, h, size, generator=g) * a, bf) for h, size, a in ((heads, dim, 1.0), (kv_heads, dim, 1.5), (kv_heads, value_dim, 1.0)))
        k[n // 2] *= 8.0  # (exact in bfloat16)
        for p in range(n):
            k_pool[table[i, p // 64], :, p % 64] = k[p].to(bf).to(cuda_device)
            v_pool[table[i, p // 64], :, p % 64] = v[p].to(bf).to(cuda_device)
        seen = pr.window_visible(n, window)
        want = torch.stack([pr.softmax_sum(q[:, h] @ k[:, h * kv_heads // heads].T * scale, seen, v[:, h * kv_heads // heads]) for h in range(heads)], 1)
        wants.append(want[n - count:].reshape(count, -1))
        qs.append(q[n - count:].reshape(count, -1))
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=cuda_device)  # noqa: E731
    rows = torch.cat(qs).to(bf).to(cuda_device)
    out = torch.full((rows.shape[0], heads * value_dim), float("nan"), dtype=bf, device=cuda_device)
    cu = i32(np.concatenate([[0], np.cumsum(counts)]).tolist())
    ops.gated_attention(rows, out, k_pool, v_pool, table.to(cuda_device), cu, i32(lengths), max(counts), heads, kv_heads, dim, value_dim, "softmax",
                        scale, window=window or 0, kernel="tcgen05")
    assert scaled_error(out.double().cpu(), torch.cat(wants)) < 6e-3
    other = torch.empty_like(out)
    ops.gated_attention(rows, other, k_pool, v_pool, table.to(cuda_device), cu, i32(lengths), max(counts), heads, kv_heads, dim, value_dim, "softmax",
                        scale, window=window or 0, kernel="rows")
    assert scaled_error(out.double().cpu(), other.double().cpu()) < 6e-3


@pytest.mark.parametrize("heads,dim,rot,value_dim,gated", [(3, 64, 64, 128, True), (2, 48, 16, 40, True), (4, 64, 0, 64, False), (1, 128, 64, 128, True),
                                                           (2, 8, 8, 8, True), (2, 96, 104, 72, False)])
def test_prompt_attention_on_its_own_rows(cuda_device, heads, dim, rot, value_dim, gated):
    """Prompts of unequal lengths that start their sequences; rows behind the last sequence hold NaN (they belong to nobody), columns of
    padding hold zeros in keys and values and anything finite in the queries; a gate per head."""
    from models_b200.kernels import ops

    g = torch.Generator().manual_seed(dim + rot)
    whole = lambda n: -(-n // 64) * 64  # noqa: E731
    bf, lengths = torch.bfloat16, [70, 1, 300, 64, 33]
    T = sum(lengths)
    spare = 20
    KD, RD, VD = whole(dim), whole(rot), whole(value_dim)
    scale = 1.3 * (dim + rot) ** -0.5
    q = _rounded(torch.randn(T, heads, dim + rot, generator=g), bf)
    k, v, r = (_rounded(torch.randn(*s, generator=g), bf) for s in ((T, heads, dim), (T, heads, value_dim), (T, rot)))
    gate = _rounded(torch.randn(T, heads, generator=g), bf)
    wants, at = [], 0
    for n in lengths:
        s = slice(at, at + n)
        score = [(q[s, h, :dim] @ k[s, h].T + q[s, h, dim:] @ r[s].T) * scale for h in range(heads)]
        one = torch.stack([pr.softmax_sum(score[h], pr.window_visible(n, None), v[s, h]) for h in range(heads)], 1)
        wants.append((one * torch.sigmoid(gate[s])[:, :, None] if gated else one).reshape(n, -1))
        at += n
    nan = lambda *shape: torch.full(shape, float("nan"), dtype=bf, device=cuda_device)  # noqa: E731

    def rows(t, size, heads=heads):  # [T, heads, n] -> [T + spare, heads * size], zeros in the padding, NaN behind
        out = nan(T + spare, heads * size)
        padded = torch.zeros(T, heads, size, dtype=F)
        padded[:, :, :t.shape[-1]] = t
        out[:T] = padded.reshape(T, -1).to(bf).to(cuda_device)
        return out

    kv = torch.cat([rows(k, KD), rows(v, VD)], dim=1).contiguous()
    q_rows = nan(T + spare, heads * (dim + rot))
    q_rows[:T] = q.reshape(T, -1).to(bf).to(cuda_device)
    out = torch.full((T + spare, heads * value_dim + 8), 7.0, dtype=bf, device=cuda_device)
    gates = nan(T + spare, heads)
    gates[:T] = gate.to(bf).to(cuda_device)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=cuda_device)  # noqa: E731
    ops.prompt_attention(q_rows, rows(q[..., dim:], RD) if rot else None, kv[:, :heads * KD], kv[:, heads * KD:],
                         rows(r[:, None], RD, 1) if rot else None, out[:, :heads * value_dim],
                         i32(np.concatenate([[0], np.cumsum(lengths)]).tolist()), i32(lengths), max(lengths), heads, dim + rot, value_dim, scale,
                         gates if gated else None)
    assert scaled_error(out[:T, :heads * value_dim].double().cpu(), torch.cat(wants)) < 6e-3
    assert bool((out[T:] == 7).all()) and bool((out[:, heads * value_dim:] == 7).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,rot,interleaved", [(20, 4, 128, 64, False), (96, 16, 128, 128, False), (3, 1, 24, 8, True), (5, 5, 10, 6, False),
                                                                (4, 2, 16, 16, True), (2, 1, 40, 0, False), (6, 3, 32, 8, False)])
def test_whole_projections_normed_rotated_and_stored(cuda_device, heads, kv_heads, dim, rot, interleaved, dtype):
    """The kernel alone, in its wide and its element-wise form, up to rows of 14,336 numbers; the values are the keys' own columns."""
    from models_b200.kernels import ops

    g = torch.Generator().manual_seed(heads)
    td, T, q_width, k_width = TORCH[dtype], 5, heads * dim, kv_heads * dim
    rows = _rounded(torch.randn(T, q_width + k_width, generator=g) * torch.tensor([0.1, 1.0, 3.0, 1.0, 0.5])[:, None], td)
    gains = 1 + 0.3 * torch.randn(q_width + k_width, generator=g)
    positions = torch.tensor([0, 1, 70, 5, 300])
    angle = positions.double()[:, None] * torch.tensor([50.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=F)[None, :]
    table = torch.arange(301).double()[:, None] * torch.tensor([50.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=F)[None, :]
    cos, sin = (f(table).float().contiguous().to(cuda_device) if rot else None for f in (torch.cos, torch.sin))

    def expected(x, gain, count):
        y = (pr.over_rms(x, 1e-4) * gain.double()).view(T, count, dim)
        c, s = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
        u, v = (y[..., 0:rot:2], y[..., 1:rot:2]) if interleaved else (y[..., :rot // 2], y[..., rot // 2:rot])
        a, b = u * c - v * s, v * c + u * s
        turned = torch.stack([a, b], -1).flatten(-2) if interleaved else torch.cat([a, b], -1)
        return torch.cat([turned, y[..., rot:]], -1)

    proj = rows.to(td).to(cuda_device)
    pools = [torch.full((3, kv_heads, 64, dim), float("nan"), dtype=td, device=cuda_device) for _ in range(2)]
    slots = torch.tensor([70, 64, -1, 191, 130], dtype=torch.int32, device=cuda_device)  # (the third token stores nothing)
    q, k = proj[:, :q_width], proj[:, q_width:]
    ops.project_norm_rotate_store(q, k, k, None, None, None, gains[:q_width].to(cuda_device).contiguous(), gains[q_width:].to(cuda_device).contiguous(), 1e-4,
                                  positions.to(torch.int32).to(cuda_device), cos, sin, rot, interleaved, pools[0], pools[1], slots, heads, kv_heads, dim, dim)
    bound = 2e-6 if dtype == "float32" else 5e-3
    assert scaled_error(proj[:, :q_width].double().cpu().view(T, heads, dim), expected(rows[:, :q_width], gains[:q_width], heads)) < bound
    want = expected(rows[:, q_width:], gains[q_width:], kv_heads)
    raw = rows[:, q_width:].view(T, kv_heads, dim)
    for i, slot in enumerate(slots.tolist()):
        if slot >= 0:
            for pool, w in zip(pools, (want[i], raw[i])):
                assert scaled_error(pool[slot // 64, :, slot % 64].double().cpu(), w) < bound
    assert int(torch.isnan(pools[0]).any(-1).sum()) == int(torch.isnan(pools[1]).any(-1).sum()) == kv_heads * (3 * 64 - 4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("latent_dim,turned,heads,dim", [(256, 64, 4, 64), (64, 16, 3, 48), (26, 6, 2, 10), (320, 0, 2, 64), (40, 8, 5, 8), (9, 2, 1, 6)])
def test_latent_rows_for_the_cache_and_for_the_step(cuda_device, latent_dim, turned, heads, dim, dtype):
    from models_b200.kernels import ops

    g = torch.Generator().manual_seed(latent_dim)
    td, T, padded = TORCH[dtype], 4, -(-turned // 64) * 64
    k, q = _rounded(torch.randn(T, latent_dim + turned, generator=g), td), _rounded(torch.randn(T, heads * (dim + turned), generator=g), td)
    gain, positions = 1 + 0.3 * torch.randn(latent_dim, generator=g), torch.tensor([3, 0, 90, 17])
    table = torch.arange(100).double()[:, None] * torch.tensor([30.0 ** (-2.0 * i / max(turned, 1)) for i in range(turned // 2)], dtype=F)[None, :]
    c, s = torch.cos(table)[positions], torch.sin(table)[positions]

    def rotated(x):  # pairs (i, i + turned / 2)
        u, v = x[..., :turned // 2], x[..., turned // 2:]
        cc, ss = (c, s) if x.dim() == 2 else (c[:, None], s[:, None])
        return torch.cat([u * cc - v * ss, v * cc + u * ss], -1)

    latent = pr.over_rms(k[:, :latent_dim], 1e-4) * gain.double()
    tail, q_tail = rotated(k[:, latent_dim:]), rotated(q.view(T, heads, dim + turned)[..., dim:])
    bound = 2e-6 if dtype == "float32" else 5e-3
    dev = lambda t: t.to(td).to(cuda_device)  # noqa: E731
    tables = tuple(f(table).float().contiguous().to(cuda_device) if turned else None for f in (torch.cos, torch.sin))
    for queries in (None, dev(q)):
        pool = torch.full((2, 1, 64, latent_dim + turned), float("nan"), dtype=td, device=cuda_device)
        slots = torch.tensor([65, -1, 0, 127], dtype=torch.int32, device=cuda_device)
        more = {} if queries is None else {"q": queries, "heads": heads, "head_columns": dim + turned, "padded": padded}
        own, own_tail, own_q = ops.latent_rows(dev(k), gain.to(cuda_device), turned, *tables, positions.to(torch.int32).to(cuda_device), 1e-4, pool, slots, **more)
        for i, slot in enumerate(slots.tolist()):
            if slot >= 0:
                assert scaled_error(pool.view(-1, latent_dim + turned)[slot].double().cpu(), torch.cat([latent[i], tail[i]])) < bound
        assert int(torch.isnan(pool).any(-1).sum()) == 2 * 64 - 3
        if queries is not None:
            assert scaled_error(own.double().cpu(), latent) < bound
            if turned:
                assert scaled_error(own_tail[:, :turned].double().cpu(), tail) < bound and bool((own_tail[:, turned:] == 0).all())
                got = own_q.view(T, heads, padded)
                assert scaled_error(got[..., :turned].double().cpu(), q_tail) < bound and bool((got[..., turned:] == 0).all())


CUTS = ([200], [2, 60, 1, 77, 60], [70] + [1] * 130)
MIXERS = {
    "latent-small": latent(4, 16, 8, 8, 32, 0.3, 10000.0, 0), "latent-cores": latent(2, 64, 16, 32, 112, 0.11, 20000.0, 0),
    "latent-odd": latent(3, 10, 6, 14, 26, 0.24, 500.0, 0), "latent-wide": latent(8, 32, 64, 48, 256, 0.1, 900.0, 0),
    "latent-many": latent(17, 16, 16, 16, 64, 0.2, 100.0, 0), "latent-equal": latent(4, 32, 32, 64, 64, 0.12, 20000.0, 0),
    "attention-small": attention(4, 2, 16, 0.3, 9, (8, 500.0, STRETCHED), 0), "attention-cores": attention(8, 2, 64, 0.12, 70, (32, 20000.0, STRETCHED), 0),
    "attention-whole": attention(4, 4, 128, 0.09, 64, (128, 20000.0, (4.0, 1.0, 4.0, 100)), 0), "attention-one": attention(3, 1, 32, 0.2, 65, None, 0),
    "attention-odd": attention(5, 5, 10, 0.35, 100, (6, 100.0, None), 0), "attention-open": attention(2, 1, 48, 0.15, None, (48, 700.0, STRETCHED), 0),
    "attention-single": attention(2, 2, 16, 0.3, 1, (16, 700.0, None), 0),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MIXERS))
def test_mixer_alone_whole_and_in_pieces(cuda_device, name, dtype):
    """A prompt whole; the same tokens as portions of 2, 60, 1 and more; and most of them one by one."""
    layer = MIXERS[name]
    spec = _spec_of(layer).mixer
    normal = lambda a, b=0.0: lambda s, g: torch.randn(s, generator=g) * a + b  # noqa: E731
    w = _weights(_shapes(spec), 5, 0.25, norm=normal(0.25, 1.2), q=normal(0.4), k=normal(0.4), uk=normal(0.4))
    part = _part("mixer", spec, w, dtype, cuda_device)
    h = _rounded(torch.randn(200, 48, generator=torch.Generator().manual_seed(9)), TORCH[dtype])
    want = pr.MIXERS[layer["type"]](h, w, "l0.mix.", layer["mixer"], 1e-5)
    for cuts in CUTS:
        assert _close(_run_in_pieces(part, h, cuts, dtype, cuda_device), want, dtype), len(cuts)


def _without(columns, directions):
    """The columns of a matrix with their parts along the given directions taken out."""
    q, _ = torch.linalg.qr(torch.stack(directions, dim=1).double())
    return (columns.double() - q @ (q.T @ columns.double())).float()


def _marked_attention(dim, window, loud, T=330, W=48, H=2):
    """Weights and rows of a windowed attention in which the last three queries ask for ONE position's key: channel 0 of a row makes its
    key, channel 1 asks for that key, and no other row's key has a part along it."""
    layer = attention(H, H, dim, 10.0 / dim, window, None, 0)
    g = torch.Generator().manual_seed(dim + loud)
    w = _weights(_shapes(_spec_of(layer).mixer), 7, 0.25, norm=lambda s, g: torch.full(s, 2.0))
    key = torch.randn(H * dim, generator=g)
    for name in ("q", "k"):
        heads = [_without(w["l0.mix." + name][h * dim:(h + 1) * dim], [key[h * dim:(h + 1) * dim]]) for h in range(H)]
        w["l0.mix." + name] = torch.cat(heads)
        w["l0.mix." + name][:, :2] = 0.0
    w["l0.mix.k"][:, 0] = w["l0.mix.q"][:, 1] = key
    h = torch.randn(T, W, generator=g) * 0.5
    h[:, :2] = 0.0
    h[loud, 0], h[T - 3:, 1] = 6.0, 6.0
    return layer, {n: t.to(torch.bfloat16).float() for n, t in w.items()}, h


def _moved(plain, w, layer, h, loud):
    """How far the last row's result moves, against its size, when the marked row loses its mark."""
    want, unmarked = plain(h, w, "l0.mix.", layer["mixer"], 1e-5)[-1], h.clone()
    unmarked[loud, 0] = 0.0
    return float((plain(unmarked, w, "l0.mix.", layer["mixer"], 1e-5)[-1] - want).abs().max() / want.abs().max())


EDGES = [(64, 63), (64, 64), (65, 64), (65, 65), (72, 71), (72, 72), (300, 299), (300, 300), (2, 1), (2, 2), (None, 329), (None, 5)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64, 128, 10])
@pytest.mark.parametrize("window,back", EDGES)
def test_one_loud_position_at_the_windows_edge(cuda_device, window, back, dim, dtype):
    """The last query follows the position it asks for when the window just holds it, and knows nothing of it when it does not: in
    a prompt, in a portion, and decoded."""
    T = 330
    loud = T - 1 - back
    layer, w, h = _marked_attention(dim, window, loud)
    h = _rounded(h, TORCH[dtype])
    moved = _moved(pr.attention, w, layer, h, loud)
    assert moved > 0.5 if window is None or back < window else moved == 0.0
    part = _part("mixer", _spec_of(layer).mixer, w, dtype, cuda_device)
    want = pr.attention(h, w, "l0.mix.", layer["mixer"], 1e-5)
    for cuts in ([T], [T - 40, 40], [T - 1, 1], [T - 3, 2, 1]):
        assert _close(_run_in_pieces(part, h, cuts, dtype, cuda_device), want, dtype), cuts


def _marked_latent(sizes, loud, T=330, W=48):
    """The same for a latent attention: the marked row's latent expands, head by head, into the key the last queries ask for."""
    H, D, R, Dv, K = sizes
    layer = latent(H, D, R, Dv, K, 1.0, 1e6, 0)
    w = _weights(_shapes(_spec_of(layer).mixer), 3, 0.15, norm=lambda s, g: torch.ones(s))
    g = torch.Generator().manual_seed(loud + K)
    direction = torch.randn(K, generator=g)
    up = w["l0.mix.uk"].view(H, D, K)
    keys = up @ (direction / direction.pow(2).mean().sqrt())
    w["l0.mix.dkv"][:K] = _without(w["l0.mix.dkv"][:K], [up[i].T @ keys[i] for i in range(H)])
    for name in ("q", "dkv", "g"):
        w["l0.mix." + name][:, :2] = 0.0
    w["l0.mix.dkv"][:K, 0] = direction
    w["l0.mix.q"].view(H, D + R, W)[:, :D, 1] = 30.0 * keys / keys.pow(2).sum(1, keepdim=True)
    h = torch.randn(T, W, generator=g) * 0.5
    h[:, :2] = 0.0
    h[loud, 0], h[T - 3:, 1] = 6.0, 1.0
    return layer, {n: t.to(torch.bfloat16).float() for n, t in w.items()}, h


LATENTS = [(4, 16, 8, 8, 32), (2, 64, 16, 32, 112), (9, 48, 16, 32, 64), (3, 10, 6, 14, 26)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", LATENTS)
@pytest.mark.parametrize("loud", [0, 1, 63, 64, 65, 300])
def test_one_loud_latent_row_far_away(cuda_device, loud, sizes, dtype):
    """One position's latent row is what the last tokens ask for: they follow it from anywhere."""
    layer, w, h = _marked_latent(sizes, loud)
    h = _rounded(h, TORCH[dtype])
    assert _moved(pr.latent_attention, w, layer, h, loud) > 0.3
    part = _part("mixer", _spec_of(layer).mixer, w, dtype, cuda_device)
    want = pr.latent_attention(h, w, "l0.mix.", layer["mixer"], 1e-5)
    T = h.shape[0]
    for cuts in ([T], [T - 40, 40], [T - 2, 2], [T - 3, 1, 1, 1]):
        assert _close(_run_in_pieces(part, h, cuts, dtype, cuda_device)[T - 3:], want[T - 3:], dtype), cuts


# ----------------------------------------------------------------------------------- whole models

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(RLX))
def test_whole_prompt_every_position(cuda_device, folders, name, dtype):
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], dtype)
    for n, seed in ((1, 1), (2, 5), (7, 2), (70, 3), (200, 4)):
        tokens = random_tokens(RLX[name]["vocab"], n, seed)
        slot = engine.open_slot()
        logits = engine.step([StepEntry(slot, tokens, list(range(n)))])
        engine.release_slot(slot)
        assert _close(logits, plain_logits(folders[name], tokens), dtype), (name, dtype, n)
    engine.cache.check()


@pytest.mark.parametrize("name", sorted(RLX))
def test_residual_stream_after_every_layer(cuda_device, folders, name):
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], "float32")
    tokens = random_tokens(RLX[name]["vocab"], 90, 6)
    seen = []
    engine.model.observer = lambda run, x: seen.append(x.double().cpu())
    slot = engine.open_slot()
    engine.step([StepEntry(slot, tokens, [89])])
    expected = []
    plain_logits(folders[name], tokens, expected)
    assert len(seen) == len(expected) == len(pr.run_order(RLX[name]))
    for run, (got, want) in enumerate(zip(seen, expected)):
        assert scaled_error(got, want) < 2e-5, run


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(RLX))
def test_prompt_then_token_by_token(cuda_device, folders, name, dtype):
    """A short prompt, then 130 tokens one by one: the decode form of the attention crosses cache pages and windows (pages behind
    the widest window are given back); a looped layer's passes each read the rows they wrote themselves."""
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], dtype)
    n, head = 150, 20
    tokens = random_tokens(RLX[name]["vocab"], n, 7)
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
    tokens = random_tokens(RLX[name]["vocab"], 70, 17)
    expected = plain_logits(folders[name], tokens)
    slot = engine.open_slot()
    rows = [engine.step([StepEntry(slot, [t], [0])]) for t in tokens]
    assert _close(torch.cat(rows), expected, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,portions", [("A", [2, 3, 17, 64, 1, 2, 90, 21]), ("B", [64, 64, 2, 70]), ("C", [130, 2, 68, 200]), ("D", [5, 2, 2, 129, 62])])
def test_prompt_in_portions(cuda_device, folders, name, portions, dtype):
    """A portion starts inside a sequence: its queries see the window's earlier rows, and every earlier latent row."""
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], dtype)
    tokens = random_tokens(RLX[name]["vocab"], sum(portions), 8)
    expected = plain_logits(folders[name], tokens)
    slot = engine.open_slot()
    at, rows = 0, []
    for count in portions:
        rows.append(engine.step([StepEntry(slot, tokens[at:at + count], list(range(count)))]).clone())
        at += count
    assert _close(torch.cat(rows), expected, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(RLX))
def test_unequal_batches_and_slots_used_again(cuda_device, folders, name, dtype):
    """Four prompts of unequal lengths in one step, decoded together while the shorter ones end; then new requests take the freed
    slots and pages (their pages hold old rows)."""
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], dtype, max_tokens=1024)
    vocab = RLX[name]["vocab"]
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
    and another takes its slot (and must not inherit its rows)."""
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], dtype, max_tokens=4096)
    engine.enable_decode_graphs(4)
    vocab = RLX[name]["vocab"]
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
@pytest.mark.parametrize("name", sorted(RLX))
def test_prompt_steps_and_decode_steps_from_captures(cuda_device, folders, name, dtype):
    """Prompts of one length class four times over (short prompt steps are captured too), then tokens one by one, and two sequences
    side by side, from captured decode steps."""
    from models_b200.engine import StepEntry

    engine = _engine(folders[name], dtype, 2048)
    engine.enable_decode_graphs(4)
    vocab = RLX[name]["vocab"]
    other = random_tokens(vocab, 60, 99)
    other_want = plain_logits(folders[name], other)
    for seed in range(4):
        tokens = random_tokens(vocab, 130, seed)
        want = plain_logits(folders[name], tokens)
        slot, beside = engine.open_slot(), engine.open_slot()
        rows = [engine.step([StepEntry(slot, tokens[:100], [0, 99])]).clone()]
        side = [engine.step([StepEntry(beside, other[:40], [39])]).clone()]
        for i in range(10):
            rows.append(engine.decode([slot], [tokens[100 + i]]).clone())
        for i in range(20):
            both = engine.decode([beside, slot], [other[40 + i], tokens[110 + i]])
            side.append(both[:1].clone())
            rows.append(both[1:].clone())
        assert _close(torch.cat(rows), torch.cat([want[:1], want[99:]]), dtype), seed
        assert _close(torch.cat(side), other_want[39:], dtype), seed
        engine.release_slot(slot)
        engine.release_slot(beside)
    engine.cache.check()


@pytest.mark.parametrize("rows", [2, 8, 12, 40])
def test_decoding_batches_of_every_product_form(cuda_device, folders, rows):
    """So many sequences decoded together that every form of the decode products runs: few rows, and rows on the wide tiles."""
    from models_b200.engine import StepEntry

    for name in ("A", "C"):
        engine = _engine(folders[name], "bfloat16", 4096, max_slots=48)
        vocab = RLX[name]["vocab"]
        full = [random_tokens(vocab, 6 + i % 5, 200 + i) for i in range(rows)]
        wanted = [plain_logits(folders[name], t) for t in full]
        slots = [engine.open_slot() for _ in full]
        engine.step([StepEntry(s, t[:2], []) for s, t in zip(slots, full)])
        got, want = [], []
        for at in range(2, 6):
            out = engine.step([StepEntry(s, [t[at]], [0]) for s, t in zip(slots, full)])
            got.append(out.clone())
            want.append(torch.stack([w[at] for w in wanted]))
        assert _close(torch.cat(got), torch.cat(want), "bfloat16"), name
        for s in slots:
            engine.release_slot(s)


RLX_MID = model(1000, 384, 1e-6, 0.8, (1, 3, 2), [
    attention(6, 3, 64, 0.14, 96, (40, 30000.0, (6.0, 1.0, 4.0, 200)), 320, 0.9),
    latent(6, 48, 32, 80, 176, 0.11, 30000.0, 200, 2.0),
    attention(3, 1, 128, 0.09, 250, (128, 8000.0, None), 448, 1.5),
    latent(10, 64, 64, 64, 96, 0.09, 700.0, 0),
])


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_mid_sized_model_long_prompts_and_batches(cuda_device, tmp_path, dtype):
    """Sizes between the small configurations and the benchmark's: a prompt of 700 tokens whole, then decoded across window edges;
    three unequal prompts in one step (1, 300 and 650 tokens), then decoded together while the short one ends."""
    from models_b200.engine import StepEntry

    folder = make_folder(RLX_MID, 77, tmp_path)
    engine = _engine(folder, dtype, max_tokens=4096)
    vocab = RLX_MID["vocab"]
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
        vocab = RLX[name]["vocab"]
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
    prompts = [random_tokens(RLX["A"]["vocab"], n, 50 + n) for n in (3, 40, 11)]
    steps = 40
    config, weights = pr.read_model_folder(folder)
    expected, margins = [], []
    for prompt in prompts:
        tokens, out, margin = list(prompt), [], []
        for _ in range(steps):
            logits = pr.forward(config, weights, tokens)[-1]
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
    """bin/trace_run on a Rulunex folder: two prompts in one step, then decoded together from captured steps."""
    name = "D"
    vocab = RLX[name]["vocab"]
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
