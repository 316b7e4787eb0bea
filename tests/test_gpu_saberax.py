"""Saberax on the GPU against the plain implementation: every kernel alone, each mixer alone over
requests cut into portions (also with inputs made so that one key or the sink carries the answer), whole
prompts, the same requests cut in different ways, long decoding, reused pages and state slots, and greedy
generation through the entry point.

float32 is the sharp comparison: a mechanism alone agrees to 2e-5 of its largest output, the whole
model to 6e-5 of the largest logit.  In bfloat16 a mechanism alone agrees to 3e-2; in the whole model
an expert chosen differently moves a row, so the bound is 3e-2 for half the rows and 0.12 for nine out
of ten."""
import copy
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import pytest
import torch

import plain_saberax as plain
import traces
from saberax_util import (SMALL, attention, dense, make_drawn_model, make_model, mixer_weights, mlp_weights, moe, norm_weights,
                          rising, windowed)
from test_gpu_feruzen import MODEL_RTOL, _compare, _run, _run_mixer
from test_gpu_ruvuvik import _paged
from util import assert_close_logits, random_tokens

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64
DTYPES = [torch.float32, torch.bfloat16]
LENGTHS = {"A": [70, 45, 120, 33, 17, 2, 64, 1], "B": [40, 9, 130, 1], "C": [300, 33, 150, 64, 217, 17]}


@pytest.fixture(scope="module")
def ops():
    from tinyinfer_b200.kernels import cuda_ops
    return cuda_ops(DEV)


def _requests(name):
    return {f"r{i}": random_tokens(SMALL[name]["vocab"], n, seed=700 + i) for i, n in enumerate(LENGTHS[name])}


_PLAIN = {}


def _plain(model_dir, name):
    if name not in _PLAIN:
        cfg, w = plain.load_folder(model_dir)
        _PLAIN[name] = {r: plain.forward(cfg, w, t) for r, t in _requests(name).items()}
    return _PLAIN[name]


def _close(got, want, dtype, what):
    tol = 2e-5 if dtype == torch.float32 else 3e-2
    err = (got.double().cpu() - want).abs().max() / want.abs().max()
    assert err < tol, f"{what}: off by {float(err):.3g} of the largest value"


# ---- kernels alone ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(1, 36), (9, 48), (5, 250), (3, 1024), (4, 2048), (2, 5120), (3, 9000), (1100, 96), (1030, 1000),
                                   (1027, 2048), (1025, 3072)])
def test_layer_norm(ops, sizes, dtype):
    """Rows whose mean is far larger than their spread among them: the deviations are taken first."""
    t, n = sizes
    g = torch.Generator().manual_seed(n)
    x = torch.randn((t, n), generator=g) * torch.logspace(-1, 1, t)[:, None] + torch.randn((t, 1), generator=g) * 30
    w, b = 1 + 0.3 * torch.randn((n,), generator=g), torch.randn((n,), generator=g)
    want = plain.layer_norm(x.double(), w.double(), b.double(), 1e-5)
    out = torch.empty((t, n), dtype=dtype, device=DEV)
    ops.layer_norm(x.to(DEV), w.to(DEV), b.to(DEV), 1e-5, out)
    _close(out, want, torch.bfloat16 if dtype == torch.bfloat16 else torch.float32, "rows")
    pick = torch.tensor([t - 1, 0, t // 2], dtype=torch.int32)
    out = torch.empty((3, n), dtype=dtype, device=DEV)
    ops.layer_norm(x.to(DEV), w.to(DEV), b.to(DEV), 1e-5, out, rows=pick.to(DEV))
    _close(out, want[pick.long()], torch.bfloat16 if dtype == torch.bfloat16 else torch.float32, "gathered rows")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(1, 36), (9, 48), (5, 250), (3, 1024), (2, 5120), (3, 9000), (1100, 96), (1030, 1000), (1027, 2048)])
def test_two_normed_rows_into_the_residual(ops, sizes, dtype):
    t, n = sizes
    g = torch.Generator().manual_seed(n)
    rand = lambda *s: torch.randn(s, generator=g)
    a, b, x = rand(t, n) * 3, rand(t, n) * torch.logspace(-2, 1, t)[:, None], rand(t, n + 4)
    wa, wb, w, bias = 1 + 0.3 * rand(n), rand(n), 1 + 0.3 * rand(n), rand(n)
    d = lambda v: v.double()
    want = d(x[:, :n]) - 0.35 * (plain.unit_rms(d(a), 1e-5) * d(wa) + plain.unit_rms(d(b), 1e-5) * d(wb))
    for then in (False, True):
        wide = x.to(DEV)
        res = wide[:, :n]
        out = torch.empty((t, n), dtype=dtype, device=DEV)
        ops.norm_sum(a.to(DEV), b.to(DEV), wa.to(DEV), wb.to(DEV), 1e-5, res, -0.35,
                     (w.to(DEV), bias.to(DEV), 1e-4, out) if then else None)
        _close(res, want, torch.float32, "residual")
        assert torch.equal(wide[:, n:].cpu(), x[:, n:])
        if then:
            _close(out, plain.layer_norm(want, d(w), d(bias), 1e-4), dtype, "normed rows")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(1, 48, 32), (5, 40, 24), (8, 1024, 256), (3, 4096, 512), (17, 130, 96), (64, 256, 4096), (90, 256, 128),
                                   (513, 1024, 320), (300, 300, 64), (2000, 512, 192), (129, 6144, 4096), (40, 5120, 4096)])
def test_products_with_a_factor(ops, sizes, dtype):
    """``x += scale (a w^T)`` for the sizes that every form of the product takes."""
    from tinyinfer_b200.parts.base import GatedSum
    t, n, k = sizes
    g = torch.Generator().manual_seed(t + n)
    a = torch.randn((t, k), generator=g).to(dtype)
    w = (torch.randn((n, k), generator=g) / k ** 0.5).to(torch.bfloat16)
    x = torch.randn((t, n), generator=g)
    y = a.double() @ w.double().T
    d = x.to(DEV)
    ops.linear(a.to(DEV), w.to(DEV), GatedSum(d, None, None, -0.7), accumulate=True, may_defer=True)
    ops.flush()
    ops.check_status()
    assert (d.cpu().double() - (x.double() - 0.7 * y)).abs().max() < 1e-4 * y.abs().max()
    d = x.to(DEV)
    ops.gated_add(y.float().to(DEV), GatedSum(d, None, None, -0.7))
    _close(d, x.double() - 0.7 * y, torch.float32, "added")


@pytest.mark.parametrize("sizes", [(1, 64, 48, 40, 96), (8, 1024, 3072, 1024, 2048), (3, 96, 64, 2080, 32), (33, 128, 512, 256, 64),
                                   (64, 40, 40, 64, 1056), (2, 48, 48, 40, 64)])
def test_two_products_of_unequal_depth_in_one_launch(ops, sizes):
    t, n1, n2, k1, k2 = sizes
    g = torch.Generator().manual_seed(n1)
    rand = lambda *s: (torch.randn(s, generator=g) / s[-1] ** 0.5).to(torch.bfloat16).to(DEV)
    a1, a2, w1, w2 = rand(t, k1), rand(t, k2), rand(n1, k1), rand(n2, k2)
    empty = lambda n: torch.full((t, n), float("nan"), dtype=torch.float32, device=DEV)
    outs = {}
    try:
        for pair in (False, True):
            ops.pair_few_rows = pair
            outs[pair] = empty(n1), empty(n2)
            before = ops.launches
            ops.linear(a1, w1, outs[pair][0], may_pair=True)
            ops.linear(a2, w2, outs[pair][1])
            ops.flush()
            assert ops.launches - before == (1 if pair and k1 % 32 == k2 % 32 == 0 else 2)
    finally:
        ops.pair_few_rows = True
    assert all(torch.equal(x, y) for x, y in zip(outs[False], outs[True]))
    _close(outs[True][1], (a2.double() @ w2.double().T).cpu(), torch.float32, "second product")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(1, 48, 40), (9, 36, 31), (70, 128, 192), (300, 64, 96), (3, 40, 24), (5, 64, 96), (40, 128, 64), (150, 72, 33),
                                   (700, 256, 1024)])
def test_feed_forward_without_a_gate(ops, sizes, dtype):
    from tinyinfer_b200.parts.base import GatedSum
    t, width, ff = sizes
    g = torch.Generator().manual_seed(ff)
    h = (torch.randn((t, width), generator=g) * 1.5).to(dtype)
    up, down = ((torch.randn(s, generator=g) / s[1] ** 0.5).to(torch.bfloat16) for s in ((ff, width), (width, ff)))
    y = torch.empty((t, ff), dtype=dtype, device=DEV)
    ops.linear_unary(h.to(DEV), up.to(DEV), "relu2", y)
    act = plain.relu_squared(h.double() @ up.double().T)
    _close(y, act, dtype, "activation")
    res = torch.zeros((t, width), dtype=torch.float32, device=DEV)
    ops.unary_ffn(h.to(DEV), up.to(DEV), down.to(DEV), GatedSum(res, None, None, 0.5), "relu2")
    ops.check_status()
    _close(res, 0.5 * act @ down.double().T, dtype, "feed-forward")


def _head_case(geom):
    heads, kv, dk, dv, rot, ps, kind = geom
    from tinyinfer_b200.parts.rope import NoPosition, RopeStretched, RopeWavelength
    if rot == 0:
        return NoPosition(), [], "halves", 1.0
    if kind == "halves":
        s = {"factor": 8.0, "original": 64, "low": 1.0, "high": 4.0}
        return RopeWavelength(dk, 777.0, 8.0, 64, 1.0, 4.0, rot), plain.wavelength_frequencies(777.0, rot, s), kind, 1.0
    s = {"factor": 4.0, "original": 128, "fast": 16.0, "slow": 1.0}
    return RopeStretched(dk, 777.0, 4.0, 128, 16.0, 1.0, rot), plain.yarn_frequencies(777.0, rot, s), kind, plain.yarn_multiplier(s)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("geom", [(4, 2, 12, 8, 8, 8, "halves"), (1, 1, 16, 16, 16, 16, "neighbours"), (6, 3, 10, 24, 0, 16, "halves"),
                                  (8, 1, 80, 64, 40, 16, "halves"), (3, 3, 7, 5, 2, 16, "neighbours"), (5, 1, 9, 9, 6, 16, "halves"),
                                  (32, 8, 128, 128, 32, 16, "neighbours"), (9, 3, 64, 64, 64, 16, "halves"), (2, 2, 256, 48, 128, 32, "neighbours"),
                                  (2, 1, 600, 20, 600, 16, "halves")])
@pytest.mark.parametrize("options", ["norm first, factor", "bias, norm last", "values from keys, norm last", "all"])
def test_heads_one_by_one(ops, geom, options, dtype):
    """Biases, the norm in front of the turn and the one behind it, the turn with its factor, queries times a factor of
    their position, values that are the projected keys; far and near positions, few tokens and many."""
    heads, kv, dk, dv, rot, ps, _ = geom
    part, freq, pairs, mult = _head_case(geom)
    from_keys = "values" in options or options == "all"
    dv = dk if from_keys else dv
    for ctx, ql in (([37, 5, 4000], [9, 5, 1]), ([300], [290])):
        step, cache, bt, positions, req = _paged(ctx, ql, ps, kv * (dk + dv), dtype)
        g = torch.Generator().manual_seed(3)
        t = len(positions)
        nq, nk, nv = heads * dk, kv * dk, 0 if from_keys else kv * dv
        proj = torch.randn((t, nq + nk + nv + 4), generator=g) * torch.logspace(-1, 1, nq + nk + nv + 4)[None]
        bias = torch.randn((nq + nk + nv,), generator=g) if "bias" in options or options == "all" else None
        first, last = "first" in options or options == "all", "last" in options or options == "all"
        qw, kw = 1 + 0.3 * torch.randn((dk,), generator=g), 1 + 0.3 * torch.randn((dk,), generator=g)
        factor = (0.7, 11) if "factor" in options or options == "all" else None
        q_out = torch.empty((t, nq), dtype=dtype, device=DEV)
        dev = lambda v: None if v is None else v.to(DEV)
        ops.heads_prepare_store(proj.to(DEV), part.rotation(DEV), step, cache, q_out, heads, kv, dk, dv, bias=dev(bias),
                                pre_norm=(dev(qw), dev(kw), 1e-5) if first else None, post_norm_eps=1e-5 if last else None,
                                query_factor=factor, values_from_keys=from_keys)
        ops.check_status()
        p64, pos = proj.double()[:, :nq + nk + nv], torch.tensor(positions)
        p64 = p64 if bias is None else p64 + bias.double()
        q, k = p64[:, :nq].reshape(t, heads, dk), p64[:, nq:nq + nk].reshape(t, kv, dk)
        v = k if from_keys else p64[:, nq + nk:].reshape(t, kv, dv)
        if first:
            q, k = plain.unit_rms(q, 1e-5) * qw.double(), plain.unit_rms(k, 1e-5) * kw.double()
        # the angle as the engine makes it: a float32 product of the position and the float32 frequency
        freq32 = [float(torch.tensor(f, dtype=torch.float32)) for f in freq]
        q, k = plain.turn(q, pos, freq32, pairs, mult), plain.turn(k, pos, freq32, pairs, mult)
        if last:
            q, k = plain.unit_rms(q, 1e-5), plain.unit_rms(k, 1e-5)
        if factor is not None:
            q = q * plain.temperature(positions, *factor).view(-1, 1, 1)
        tol = dtype if max(ctx) < 1000 or dtype != torch.float32 else None
        check = (lambda got, want, what: _close(got, want, tol, what)) if tol is not None else (
            lambda got, want, what: _close(got, want, torch.float32, what) if rot == 0 else
            _assert_small((got.double().cpu() - want).abs().max() / want.abs().max(), 2e-4, what))
        check(q_out.view(t, heads, dk), q, "queries")
        keys, values = [], []
        for i in range(t):
            page, slot = cache.pages[int(bt[req[i], positions[i] // ps])], positions[i] % ps
            keys.append(page[: kv * ps * dk].view(kv, ps, dk)[:, slot])
            values.append(page[kv * ps * dk:].view(kv, ps, dv)[:, slot])
        check(torch.stack(keys), k, "keys")
        _close(torch.stack(values), v, dtype, "values")


def _assert_small(err, tol, what):
    assert err < tol, f"{what}: off by {float(err):.3g} of the largest value"


@pytest.mark.parametrize("case", [(6, 2, None), (12, 3, (2, 1)), (12, 3, (3, 2)), (9, 9, (3, 3)), (40, 6, (8, 3)), (5, 1, (5, 1)),
                                  (300, 8, (10, 4)), (1, 1, (1, 1)), (256, 32, (8, 4)), (64, 4, (32, 3))])
def test_choice_by_sigmoid_scores(ops, case):
    total, top, groups = case
    g = torch.Generator().manual_seed(total * 7 + top)
    t = 133
    z = torch.randn((t, total + 3), generator=g) * 2.0
    z[5] = 0.0                                            # all scores equal: the correction alone decides
    correction = torch.randn((total,), generator=g) * 0.4 - 0.5          # most choice scores lie below zero
    ids = torch.empty((t, top), dtype=torch.int32, device=DEV)
    weights = torch.empty((t, top), dtype=torch.float32, device=DEV)
    ops.router_choose(z.to(DEV), total, top, ids, weights, correction.to(DEV), *(groups or (1, 1)), sigmoid=True, best_of=2,
                      normalize=True, factor=2.5)
    s = torch.sigmoid(z[:, :total].to(DEV)).cpu()          # the float32 scores decide
    choice = s + correction
    for i in range(t):
        want = plain.choose(choice[i].double(), top, *(groups or (1, 1)))
        gaps = sorted(choice[i].tolist())
        if min((b - a for a, b in zip(gaps, gaps[1:])), default=1.0) < 1e-6 and i != 5:
            continue                                      # a close call between two outputs
        assert ids[i].tolist() == want, f"row {i}"
        w = s[i][want].double()
        assert torch.allclose(weights[i].cpu().double(), 2.5 * w / (w.sum() + 1e-20), rtol=1e-5)
    # softmax scores and the largest value of a group stay as they were
    ops.router_choose(z.to(DEV), total, top, ids, weights, None)
    s = torch.softmax(z[:, :total].double(), dim=-1)
    assert torch.allclose(weights.cpu().double().sum(-1), s.topk(top, dim=-1).values.sum(-1), rtol=1e-5)


def test_scores_of_nothing_do_not_divide_by_zero(ops):
    z = torch.full((3, 8), -200.0, device=DEV)
    ids, weights = torch.empty((3, 2), dtype=torch.int32, device=DEV), torch.empty((3, 2), device=DEV)
    ops.router_choose(z, 8, 2, ids, weights, None, 4, 2, sigmoid=True, best_of=2, normalize=True, factor=3.0)
    assert torch.isfinite(weights).all() and ids.tolist() == [[0, 1]] * 3


# ---- parts alone ---------------------------------------------------------------------------------
def _part(ops, category, spec, w):
    from tinyinfer_b200.parts.base import build_part
    part = build_part(category, spec)
    part.load_weights({k: v.to(DEV) for k, v in w.items()}, ops)
    return part


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp", [moe(12, 3, 24, 1.7, groups=(3, 2), shared=40), moe(8, 2, 16, 2.5, groups=(2, 1)), moe(4, 4, 12, 1.0),
                                 moe(5, 1, 9, 3.0, groups=(1, 1), shared=7), moe(16, 4, 64, 2.0, groups=(4, 2), shared=128),
                                 moe(3, 2, 32, 1.5, shared=4096), dense(40), dense(192)])
@pytest.mark.parametrize("t", [1, 7, 60, 150, 700])  # 60: a shared expert beside the router; 150, 700: grouped products
def test_each_feed_forward_alone(ops, mlp, t, dtype):
    from tinyinfer_b200.config import saberax
    from tinyinfer_b200.parts.base import GatedSum
    width = 64
    g = torch.Generator().manual_seed(t)
    w = mlp_weights(mlp, width, g)
    part = _part(ops, "ffn", saberax._ffn_spec(SimpleNamespace(width=width), saberax._mlp({"mlp": mlp}, "here")), w)
    h = (torch.randn((t, width), generator=g) * 1.5).to(dtype)
    y = plain.feed_forward({k: v.double() for k, v in w.items()}, "", h.double(), mlp)
    assert part.ends_in_linear or part.takes_factor
    for factor in (1.0, -0.6):
        x = torch.zeros((t, width), dtype=torch.float32, device=DEV)
        part.forward(ops, h.to(DEV), x if factor == 1.0 else GatedSum(x, None, None, factor), SimpleNamespace(scratch={}))
        ops.flush()
        ops.check_status()
        err = (x.cpu().double() - factor * y).abs().max(dim=-1).values / y.abs().max()
        if dtype == torch.float32:
            assert err.max() < 2e-5, f"off by {float(err.max()):.3g}"
        else:                                            # a near-tie in the choice may fall the other way
            assert err.median() < 3e-2 and (t < 10 or torch.quantile(err, 0.9) < 3e-2)


MIXER_CASES = [
    attention(4, 2, 10, 19, 6, 0.6, 40.0, (8.0, 40, 1.0, 4.0)), attention(3, 1, 16, 33, 16, 0.4, 900.0, (2.0, 25, 0.5, 3.0)),
    attention(2, 2, 8, 1, 2, 1.0, 7.0, (1.0, 8, 1.0, 2.0)), attention(4, 4, 64, 20, 64, 0.2, 3e5, (8.0, 64, 1.0, 4.0)),
    attention(8, 2, 128, 50, 64, 0.1, 1e4, (4.0, 32, 1.0, 4.0)), attention(5, 5, 32, 16, 0, 0.3, 2.0, (1.0, 1, 1.0, 1.0)),
    rising(6, 3, 8, 12, 0.3, 0.4, 9, 60, 3, 3), rising(1, 1, 6, 5, 0.4, 0.0, 1, 20, 1, 1), rising(3, 3, 7, 7, 0.4, 1.5, 1, 12, 12, 6),
    rising(4, 2, 48, 32, 0.15, 0.2, 40, 192, 3, 4), rising(2, 1, 128, 64, 0.1, 1.0, 16, 128, 8, 2),
    windowed(4, 2, 12, 8, 21, 8, 0.5, 500.0, (4.0, 32, 8.0, 1.0), (3, 8, 20, 9.0)),
    windowed(1, 1, 16, 16, 1, 0, 0.25, 2.0, (1.0, 1, 1.0, 1.0), (1, 16, 16, 1.0)),
    windowed(2, 1, 9, 4, 64, 4, 0.3, 10.0, (3.0, 16, 2.0, 1.0), (1, 5, 9, 2.5)),
    windowed(4, 2, 64, 64, 17, 32, 0.125, 2e4, (4.0, 128, 16.0, 1.0), (2, 64, 128, 16.0)),
    windowed(2, 1, 128, 32, 33, 128, 0.09, 5000.0, (2.0, 256, 32.0, 1.0), (4, 32, 32, 4.0)),
    windowed(6, 3, 48, 96, 2, 16, 0.2, 100.0, (2.0, 16, 4.0, 1.0), (1, 200, 96, 2.0))]
CUTS = [[("a", 30), ("b", 1)], [("b", 2), ("c", 5)], [("a", 1), ("b", 30), ("c", 1)], [("a", 2), ("c", 1)],
        [("a", 17), ("b", 7), ("c", 33)], [("a", 1)], [("a", 1), ("c", 2)], [("b", 0), ("d", 70)], [("d", 1), ("a", 1)]]
TOTAL = {"a": 53, "b": 40, "c": 42, "d": 71}
EPS = 1e-5


def _mixer_part(ops, entry, width, w):
    from tinyinfer_b200.config import saberax
    cfg = SimpleNamespace(width=width, norm_eps=EPS)
    layer = saberax.SaberaxLayer(entry["type"], saberax._mixer(entry, "here", entry["type"]), None)
    return _part(ops, "mixer", saberax._mixer_spec(cfg, layer), w)


def _plain_mixer(entry, w, x):
    return plain.mixer({"norm": {"eps": EPS}}, {k: v.double() for k, v in w.items()}, entry, "", x)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("entry", MIXER_CASES, ids=[f"{e['type']}-{i}" for i, e in enumerate(MIXER_CASES)])
def test_each_mixer_alone_in_portions(ops, entry, dtype):
    """Four requests in portions down to one token; the fourth takes the slot that the second gave back."""
    width = 64
    g = torch.Generator().manual_seed(5)
    w = mixer_weights(entry["type"], entry["mixer"], width, g)
    part = _mixer_part(ops, entry, width, w)
    inputs = {r: torch.randn((n, width), generator=g).to(dtype).float() for r, n in TOTAL.items()}
    got = _run_mixer(ops, part, inputs, CUTS, dtype)
    for r, x in inputs.items():
        _close(got[r], _plain_mixer(entry, w, x.double()), dtype, f"{entry['type']} request {r}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("entry", [MIXER_CASES[4], MIXER_CASES[9], MIXER_CASES[14]], ids=lambda e: e["type"])
def test_mixers_over_long_portions(ops, entry, dtype):
    """Portions of more than a tile of rows between short ones; a slot that a finished request gave back starts at
    zero again."""
    width = 64
    g = torch.Generator().manual_seed(4)
    w = mixer_weights(entry["type"], entry["mixer"], width, g)
    part = _mixer_part(ops, entry, width, w)
    inputs = {"a": torch.randn((203, width), generator=g), "b": torch.randn((72, width), generator=g)}
    inputs["c"] = inputs["b"][:40] * 0.5
    cuts = [[("a", 3)], [("a", 130)], [("a", 1), ("b", 70)], [("a", 69), ("b", 2)], [("a", 0), ("c", 2)], [("c", 38)]]
    got = _run_mixer(ops, part, inputs, cuts, dtype, max_requests=2)
    for r, x in inputs.items():
        _close(got[r], _plain_mixer(entry, w, x.to(dtype).double()), dtype, f"request {r}")


def test_sides_that_are_not_projected_mixers(ops):
    """Normed sides of any kind of mixer: the same sum without the stacked products, with and without a norm behind."""
    from tinyinfer_b200.config.plan import PartSpec
    from tinyinfer_b200.parts.base import GatedSum
    from tinyinfer_b200.parts.norm import LayerNorm
    width, dtype = 64, torch.float32
    entry = rising(2, 1, 16, 16, 0.3, 0.4, 3, 32, 2, 3)
    g = torch.Generator().manual_seed(8)
    w = mixer_weights("parallel", entry["mixer"], width, g)
    together, apart = _mixer_part(ops, entry, width, w), _mixer_part(ops, entry, width, w)
    assert together.w_in is not None
    apart.w_in, cut = None, together.cut
    apart.sides["left"].w_in, apart.sides["right"].w_in = together.w_in[:cut].contiguous(), together.w_in[cut:].contiguous()
    x = {"a": torch.randn((20, width), generator=g)}
    cuts = [[("a", 11)], [("a", 1)], [("a", 8)]]
    want = _plain_mixer(entry, w, x["a"].double())
    for part in (together, apart):
        _close(_run_mixer(ops, part, x, cuts, dtype)["a"], want, dtype, "sides")
    norm = LayerNorm(width, 1e-5)
    nw = norm_weights("weight", width, g)
    norm.load_weights({k: v.to(DEV) for k, v in nw.items()}, ops)

    class Then:                                              # a part whose forward also checks the rows behind it
        cache_spec, step_lists = together.cache_spec, together.step_lists

        def forward(self, ops, h, residual, step, cache):
            rows = together.forward_then(ops, h, GatedSum(residual, None, None, 0.5), step, cache, norm)
            _close(rows, plain.layer_norm(residual.double().cpu(), nw["weight"].double(), nw["weight.b"].double(), 1e-5), dtype, "norm")

    _close(_run_mixer(ops, Then(), x, cuts, dtype)["a"], 0.5 * want, dtype, "with a factor")
    with pytest.raises(ValueError):                          # normed sides are added with one factor
        from tinyinfer_b200.parts.base import build_part
        side = PartSpec("gated_linear_recurrence", {"hidden_size": width, "width": 8, "blocks": 1, "conv_taps": 1})
        build_part("mixer", PartSpec("parallel_mixers", {"hidden_size": width, "left": side, "right": side, "left_scale": 0.5,
                                                         "right_scale": 1.0, "norm_eps": 1e-5}))


# ---- inputs made so that one key carries the answer ------------------------------------------------
def _pointing(dim, width, dv, heads=2):
    """Projections of a layer whose heads compare the first 20 input columns and read columns 40 on."""
    q, k, v = torch.zeros((heads * dim, width)), torch.zeros((dim, width)), torch.zeros((dv, width))
    for a in range(heads):                                      # the elements behind the turned ones
        q[a * dim + dim - 20:(a + 1) * dim, :20] = torch.eye(20)
    k[dim - 20:, :20] = torch.eye(20)
    v[:, 40:40 + dv] = torch.eye(dv)
    return q, k, v


def _standing_out(pos, target, width, dtype):
    """Rows in which the token ``pos`` asks for ``target``, which alone carries a one in column 40; the token right behind
    the query looks the same."""
    g = torch.Generator().manual_seed(target)
    x = torch.zeros((pos + 2, width))
    x[:, :20] = torch.nn.functional.normalize(torch.randn((pos + 2, 20), generator=g), dim=1)
    direction = torch.nn.functional.normalize(torch.randn((20,), generator=g), dim=0)
    x[:, :20] -= 0.9 * (x[:, :20] @ direction).clamp(min=0)[:, None] * direction         # no other key comes near
    x[target, :20] = x[pos, :20] = x[pos + 1, :20] = direction
    x[target, 40] = 1.0
    return x.to(dtype).float()


def _cuts(pos, decoded):
    return [[("a", pos)], [("a", 1)], [("a", 1)]] if decoded and pos else [[("a", max(1, pos - 40))], [("a", pos + 2 - max(1, pos - 40))]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decoded", [False, True])
def test_one_key_in_a_window_a_chunk_and_far_back(ops, decoded, dtype):
    """A query that points at one key alone, just inside and just outside of windows and chunks, on both sides of page
    borders, at the first tokens, hundreds of positions back, and at the token right after itself."""
    from tinyinfer_b200.config.plan import PartSpec
    width, dim, dv, ps = 64, 24, 8, 16
    q, k, v = _pointing(dim, width, dv)
    o = torch.zeros((width, 2 * dv))
    o[:2 * dv] = torch.eye(2 * dv)
    w = {"q": q, "k": k, "v": v, "o": o}
    base = {"hidden_size": width, "num_heads": 2, "num_kv_heads": 1, "head_dim": dim, "v_head_dim": dv, "qk_norm_eps": 1e-6,
            "norm_per_head": True, "head_temperature": False, "head_gate": False,
            "position": PartSpec("rope_stretched", {"head_dim": dim, "theta": 100.0, "rotary_dim": 4, "factor": 2.0, "original": 64,
                                                    "fast": 8.0, "slow": 1.0})}
    window = dict(base, norm_before=False, norm_after=True, bias=True, window=37, scale=2.0)
    causal = dict(base, position=PartSpec("none", {}), query_factor=(0.5, 64), scale=2.0)
    chunk = dict(base, norm_before=False, norm_after=True, chunk=50, scale=2.0)
    zeros = {"q.b": torch.zeros(2 * dim), "k.b": torch.zeros(dim), "v.b": torch.zeros(dv)}
    ones = {"q.norm": torch.ones(dim), "k.norm": torch.ones(dim)}
    for spec, extra, cases in (
            (window, zeros, [(700, [664, 663, 672, 687, 688, 700]), (36, [0]), (37, [0, 1]), (1, [0, 1])]),
            (chunk, {}, [(700, [700, 699]), (749, [700, 699, 703, 704]), (49, [0, 15, 16]), (50, [49, 50]), (1, [0])]),
            (causal, ones, [(700, [0, 1, 15, 16, 351, 352, 687, 688, 699, 700]), (16, [0, 15, 16])])):
        part = _part(ops, "mixer", PartSpec("chunked_attention", spec), {n: t.to(torch.bfloat16) for n, t in {**w, **extra}.items()})
        for pos, targets in cases:
            lo = plain.visible(pos, spec.get("window"), spec.get("chunk"))
            for target in targets:
                x = _standing_out(pos, target, width, dtype)
                row = _run_mixer(ops, part, {"a": x}, _cuts(pos, decoded), dtype, page_size=ps)["a"][pos]
                # the query's own key has the same direction: the two share the weight
                want = 0.0 if target < lo else 1.0 if target == pos else 0.5
                assert abs(float(row[0]) - want) < 0.04 and abs(float(row[dv]) - want) < 0.04, (spec.get("window"), pos, target, row[0])


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_sink_and_the_gate_of_a_head(ops, dtype):
    """Keys that all score zero beside a sink of ln 3 and one that vanishes; one gate half open, one open.  The chunk's
    first tokens see few keys, so the sink weighs most there."""
    from tinyinfer_b200.config.plan import PartSpec
    width, dim, chunk = 32, 16, 20
    w = {"q": torch.zeros((2 * dim, width)), "k": torch.zeros((dim, width)), "o": torch.zeros((width, 2 * dim)),
         "sink": torch.tensor([3.0, -200.0]), "g": torch.zeros((2, width))}
    w["sink"][0] = float(torch.tensor(3.0).log())
    w["k"][:4, :4] = torch.eye(4)                              # values: the projected keys, all alike
    w["o"][:2 * dim] = torch.eye(2 * dim)
    w["g"][1, 5] = 100.0
    part = _part(ops, "mixer", PartSpec("chunked_attention", {
        "hidden_size": width, "num_heads": 2, "num_kv_heads": 1, "head_dim": dim, "v_head_dim": dim, "scale": 1.0, "qk_norm_eps": 1e-6,
        "position": PartSpec("rope_wavelength", {"head_dim": dim, "theta": 100.0, "factor": 4.0, "original": 16, "low": 1.0, "high": 4.0}),
        "norm_before": False, "norm_after": True, "values_from_keys": True, "sink": True, "head_temperature": False, "chunk": chunk}),
        {n: t.float() for n, t in w.items()})
    x = torch.zeros((45, width))
    x[:, :4], x[:, 5] = 2.0, 1.0
    rows = _run_mixer(ops, part, {"a": x}, [[("a", 21)], [("a", 1)], [("a", 23)]], dtype)["a"]
    for i in range(45):
        seen = i % chunk + 1
        assert abs(float(rows[i, 0]) - 0.5 * 2.0 * seen / (seen + 3)) < 1e-2, i
        assert abs(float(rows[i, dim]) - 2.0) < 1e-2, i


# ---- whole models ---------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_whole_prompts(tmp_path_factory, name, dtype):
    d = make_model(tmp_path_factory.getbasetemp(), name)
    steps = traces.whole(_requests(name))
    out = _run(d, dtype, steps, traces.max_live_tokens(steps))
    _compare(steps, out, _plain(d, name), dtype, f"{name} whole")


def test_every_layer_against_the_plain_rows(tmp_path_factory):
    """What each layer hands on, in float32: the first that differs names the mechanism."""
    from tinyinfer_b200 import Engine, StepEntry
    for name in ("A", "B", "C"):
        d = make_model(tmp_path_factory.getbasetemp(), name)
        cfg, w = plain.load_folder(d)
        tokens = _requests(name)["r1"]
        want = []
        plain.forward(cfg, w, tokens, layers_out=want)
        eng = Engine(d, dtype="float32", page_size=16, num_pages=8, max_requests=1)
        got = []
        for block in eng.model.blocks:
            inner = block.forward
            block.forward = lambda ops, x, step, cache, inner=inner: (inner(ops, x, step, cache), got.append(x.clone()))[0]
        eng.step([StepEntry("x", tokens, [0])])
        assert len(got) == len(want) == len(cfg["layers"])
        for i, (a, b) in enumerate(zip(got, want)):
            assert (a.cpu().double() - b).abs().max() < MODEL_RTOL * b.abs().max(), f"{name}: layer {i}"


@pytest.mark.parametrize("name, family, dtype", [
    ("A", "tail", "float32"), ("A", "portions", "float32"), ("A", "mixed", "float32"), ("A", "mixed", "bfloat16"),
    ("B", "portions", "float32"), ("B", "mixed", "float32"), ("B", "tail", "bfloat16"), ("A", "pairs", "float32"),
    ("C", "tail", "float32"), ("C", "portions", "bfloat16"), ("C", "mixed", "float32"), ("C", "mixed", "bfloat16"),
    ("C", "long portions", "bfloat16"), ("C", "long portions", "float32")])
def test_cuttings_agree_with_the_plain_implementation(tmp_path_factory, name, family, dtype):
    """Prefill against token-by-token decoding, portions down to two tokens, and up to four live
    requests of unequal length in a pool so small that pages and state slots are used again."""
    d = make_model(tmp_path_factory.getbasetemp(), name)
    reqs = _requests(name)
    steps = {"tail": lambda: traces.tail_decoded(reqs, tail=40), "portions": lambda: traces.portions(reqs),
             "pairs": lambda: traces.portions(reqs, sizes=(2,)),
             "long portions": lambda: traces.portions(reqs, sizes=(150, 2, 71, 70, 128, 3)),
             "mixed": lambda: traces.mixed(reqs, seed=5)}[family]()
    out = _run(d, dtype, steps, traces.max_live_tokens(steps))
    _compare(steps, out, _plain(d, name), dtype, f"{name} {family}")


@pytest.mark.parametrize("seed", range(20))
def test_drawn_configurations(tmp_path_factory, seed):
    """Sizes, constants and the order of layers drawn from a seed: mixed batches in a small pool in float32, whole
    prompts in bfloat16."""
    d = make_drawn_model(tmp_path_factory.getbasetemp(), seed)
    cfg, w = plain.load_folder(d)
    reqs = {f"r{i}": random_tokens(cfg["vocab"], n, seed=seed * 10 + i) for i, n in enumerate([70, 45, 33, 2, 97, 1])}
    want = {r: plain.forward(cfg, w, t) for r, t in reqs.items()}
    steps = traces.mixed(reqs, seed=seed)
    _compare(steps, _run(d, "float32", steps, traces.max_live_tokens(steps)), want, "float32", f"drawn {seed} mixed")
    steps = traces.whole(reqs)
    _compare(steps, _run(d, "bfloat16", steps, traces.max_live_tokens(steps)), want, "bfloat16", f"drawn {seed} whole")


def test_one_state_slot_used_by_every_request_in_turn(tmp_path_factory):
    d = make_model(tmp_path_factory.getbasetemp(), "A")
    steps = traces.portions(_requests("A"), sizes=(40, 2, 9))
    out = _run(d, "float32", steps, traces.max_live_tokens(steps), max_requests=1)
    _compare(steps, out, _plain(d, "A"), "float32", "one slot")


@pytest.mark.parametrize("name", ["A", "C"])
def test_float32_cuttings_give_the_same_bits(tmp_path_factory, name):
    d = make_model(tmp_path_factory.getbasetemp(), name)
    reqs = _requests(name)
    seen = {}
    for family in (traces.whole(reqs), traces.portions(reqs), traces.mixed(reqs, seed=2)):
        out = _run(d, "float32", family, traces.max_live_tokens(family))
        for r, rows in traces.collect(family, out).items():
            for p, x in rows:
                if (r, p) in seen:
                    assert torch.equal(seen[(r, p)], x), f"request {r} position {p}"
                seen[(r, p)] = x


@pytest.mark.parametrize("name, dtype", [("A", "float32"), ("C", "bfloat16")])
def test_long_decoding(tmp_path_factory, name, dtype):
    """Tokens one by one through the decode graphs, in a batch with a request that joins and one that ends."""
    from tinyinfer_b200 import Engine, StepEntry
    d = make_model(tmp_path_factory.getbasetemp(), name)
    cfg, w = plain.load_folder(d)
    tokens = {r: random_tokens(cfg["vocab"], n, seed=77 + n) for r, n in (("x", 170), ("y", 60), ("z", 90))}
    want = {r: plain.forward(cfg, w, t) for r, t in tokens.items()}
    eng = Engine(d, dtype=dtype, page_size=16, num_pages=24, max_requests=3)
    got = {r: [] for r in tokens}
    at = {}
    for now in range(200):
        for r, start in (("x", 0), ("y", 20), ("z", 45)):
            if now == start:
                got[r].append(eng.step([StepEntry(r, tokens[r][:4], [3])])[0].cpu())
                at[r] = 4
        live = [r for r in at if at[r] < len(tokens[r])]
        if not live:
            break
        rows = eng.decode_step([StepEntry(r, [tokens[r][at[r]]], [0]) for r in live]).cpu()
        for r, row in zip(live, rows):
            got[r].append(row.clone())
            at[r] += 1
            if at[r] == len(tokens[r]):
                eng.finish(r)
        eng.cache.check()
    for r in tokens:
        if dtype == "float32":
            assert_close_logits(torch.stack(got[r]), want[r][3:], MODEL_RTOL, f"long decoding {r}")
        else:
            err = (torch.stack(got[r]).double() - want[r][3:]).abs().max(dim=-1).values / want[r].abs().max()
            assert err.median() < 3e-2 and torch.quantile(err, 0.9) < 0.12, f"{r}: {float(err.max())}"
    assert all(n == 24 for n in eng.cache.free_pages())


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_entry_point(tmp_path_factory, name, graphs):
    from tinyinfer_b200 import LLM, SamplingParams
    d = make_model(tmp_path_factory.getbasetemp(), name)
    cfg, w = plain.load_folder(d)
    prompts = [random_tokens(cfg["vocab"], n, seed=n) for n in (5, 31, 12)]
    llm = LLM(d, dtype="float32", max_seq=128, max_num_seqs=2, max_batched_tokens=24, page_size=16,
              cuda_graph=graphs)
    outs = llm.generate(prompts, SamplingParams(max_tokens=8))
    for prompt, out in zip(prompts, outs):
        assert out.tokens == plain.greedy(cfg, w, prompt, 8), f"prompt of {len(prompt)} tokens"


def test_random_weights_from_a_configuration(tmp_path):
    from tinyinfer_b200 import Engine, StepEntry, write_random_model
    cfg = copy.deepcopy(SMALL["C"])
    for entry in cfg["layers"]:
        if entry["type"] == "parallel_2":                # no stored tensor says it
            entry["mixer"]["right"]["decay_rank"] = 24
    tokens = random_tokens(cfg["vocab"], 90, seed=1)
    a = Engine(config=cfg, seed=5, dtype="bfloat16", page_size=16, num_pages=16, max_requests=2)
    la = a.step([StepEntry("a", tokens, [0, 50, 89])])
    d = os.path.join(str(tmp_path), "written")
    write_random_model(d, cfg, seed=5)
    b = Engine(d, dtype="bfloat16", page_size=16, num_pages=16, max_requests=2)
    lb = b.step([StepEntry("a", tokens, [0, 50, 89])])
    assert torch.isfinite(la).all() and torch.equal(la, lb)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_program(tmp_path_factory, tmp_path, dtype):
    """The replay program as a user starts it: steps on standard input, logits in files."""
    import numpy as np
    d = make_model(tmp_path_factory.getbasetemp(), "C")
    steps = traces.mixed(_requests("C"), seed=9)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = str(tmp_path / "out")
    proc = subprocess.run(
        [sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", out,
         "--max-tokens", str(traces.max_live_tokens(steps))],
        input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [ln for ln in proc.stdout.splitlines() if ln.startswith("done ")] == [f"done {s['step']}" for s in steps]
    vocab = SMALL["C"]["vocab"]
    outputs = {}
    for s in steps:
        wanted = sum(len(e["want"]) for e in s["entries"])
        if wanted:
            data = np.fromfile(os.path.join(out, f"{s['step']}.f32"), dtype="<f4")
            outputs[s["step"]] = torch.from_numpy(data.reshape(wanted, vocab).copy())
    _compare(steps, outputs, _plain(d, "C"), dtype, f"replay {dtype}")


def test_command_line_with_token_ids(tmp_path_factory, capsys):
    from tinyinfer_b200 import cli
    d = make_model(tmp_path_factory.getbasetemp(), "B")
    cfg, w = plain.load_folder(d)
    prompt = random_tokens(cfg["vocab"], 9, seed=4)
    rc = cli.main(["-m", d, "--tokens", "-p", " ".join(map(str, prompt)), "-n", "6", "--dtype", "float32",
                   "--max-seq", "64", "--max-num-seqs", "2", "--page-size", "16"])
    assert rc == 0
    out = capsys.readouterr().out
    line = [ln for ln in out.splitlines() if ln.startswith("[output]")][0]
    assert [int(x) for x in line.split()[1:]] == plain.greedy(cfg, w, prompt, 6)
