"""Vametar on the GPU against the plain implementation: every kernel alone, each mixer alone over
requests cut into portions (also with inputs made so that one key, one write or one channel carries
the answer), whole prompts, the same requests cut in different ways, long decoding, reused pages and
state slots, and greedy generation through the entry point.

float32 is the sharp comparison: a mechanism alone agrees to 2e-5 of its largest output, the whole
model to 6e-5 of the largest logit.  In bfloat16 a mechanism alone agrees to 3e-2."""
import copy
import json
import math
import os
import subprocess
import sys
from types import SimpleNamespace

import pytest
import torch

import plain_vametar as plain
import traces
from test_gpu_feruzen import MODEL_RTOL, _compare, _rows_step, _run, _run_mixer
from test_gpu_ruvuvik import _paged
from util import assert_close_logits, random_tokens
from vametar_util import SMALL, attention, gla, make_drawn_model, make_model, mixer_weights, mlp_weights, rglru

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64
DTYPES = [torch.float32, torch.bfloat16]
LENGTHS = {"A": [70, 45, 120, 33, 17, 2, 64, 1], "B": [40, 9, 130, 1], "C": [300, 33, 150, 64, 217, 17], "D": [50, 3, 90]}


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


def _state(floats, slots=3, dtype=torch.float32):
    return SimpleNamespace(state=torch.zeros((slots, floats), dtype=dtype, device=DEV), slots=None, writes=True)


# three requests in portions down to one row; "b" ends and "d" takes its slot
PORTIONS = [[("a", 1), ("b", 5)], [("a", 1), ("c", 2)], [("a", 2), ("b", 1), ("c", 1)], [("a", 12), ("b", 3), ("c", 11)],
            [("a", 7), ("d", 4)], [("d", 1), ("a", 1)], [("d", 2)]]
COUNTS = {"a": 24, "b": 9, "c": 14, "d": 7}
SLOT = {"a": 2, "b": 0, "c": 1, "d": 0}


def _walk(state, run):
    """``run(cut, at, step)`` for every step of ``PORTIONS``; what a request keeps is cleared where it starts."""
    at = {r: 0 for r in COUNTS}
    for cut in PORTIONS:
        for r, _ in cut:
            if at[r] == 0:
                state.state[SLOT[r]].zero_()
        step, state.slots = _rows_step([n for _, n in cut], [SLOT[r] for r, _ in cut])
        step.positions = torch.tensor([at[r] + i for r, n in cut for i in range(n)], dtype=torch.int32, device=DEV)
        run(cut, at, step)
        for r, n in cut:
            at[r] += n
    assert at == COUNTS


# ---- kernels alone ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", [(40, 37, 1009, 11), (7, 1, 0, 1), (300, 500, 3, 499), (4, 100_003, 99_998, 100_001 + 7 * 100_003)])
def test_embedding_with_a_hash_of_two_tokens(ops, case, dtype):
    width, buckets, mul_prev, mul_cur = case
    vocab = 200_000 if buckets > 1000 else 50             # the last case: products of more than 32 bits
    g = torch.Generator().manual_seed(width)
    table = torch.randn((vocab, width), generator=g).to(dtype)
    bigram = torch.randn((buckets + 1, width), generator=g).to(dtype)
    tokens = {r: random_tokens(vocab, n, seed=n) for r, n in COUNTS.items()}
    state = _state(1, dtype=torch.int32)
    got = {r: [] for r in COUNTS}

    def run(cut, at, step):
        ids = torch.tensor([x for r, n in cut for x in tokens[r][at[r]:at[r] + n]], dtype=torch.int32, device=DEV)
        out = torch.empty((len(ids), width), dtype=torch.float32, device=DEV)
        ops.embed_bigram(table.to(DEV), bigram.to(DEV), ids, buckets, mul_prev % buckets, mul_cur % buckets, step, state, out)
        o = 0
        for r, n in cut:
            got[r].append(out[o:o + n].cpu())
            o += n

    _walk(state, run)
    cfg = {"embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}
    for r in COUNTS:
        want = plain.embed(cfg, {"embed": table.double(), "bigram": bigram.double()}, tokens[r])
        assert (torch.cat(got[r]).double() - want).abs().max() < 1e-6, r


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [36, 48, 250, 1024, 2051])
def test_norm_and_token_shift_over_portions(ops, width, dtype):
    g = torch.Generator().manual_seed(width)
    x = {r: torch.randn((n, width), generator=g) * torch.logspace(-1, 1, n)[:, None] for r, n in COUNTS.items()}
    w, mu = 1 + 0.3 * torch.randn((width,), generator=g), torch.randn((width,), generator=g) * 0.7
    state = _state(width)
    plain_rows, shifted_rows = {r: [] for r in COUNTS}, {r: [] for r in COUNTS}

    def run(cut, at, step):
        rows = torch.cat([x[r][at[r]:at[r] + n] for r, n in cut]).to(DEV)
        h = torch.empty(rows.shape, dtype=dtype, device=DEV)
        s = torch.empty_like(h)
        ops.rmsnorm_shift(rows, w.to(DEV), 1e-5, mu.to(DEV), step, state, h, s)
        o = 0
        for r, n in cut:
            plain_rows[r].append(h[o:o + n].cpu())
            shifted_rows[r].append(s[o:o + n].cpu())
            o += n

    _walk(state, run)
    for r in COUNTS:
        h = plain.unit_rms(x[r].double(), 1e-5) * w.double()
        _close(torch.cat(plain_rows[r]), h, dtype, f"norm of {r}")
        _close(torch.cat(shifted_rows[r]), plain.token_shift(h, mu.double()), dtype, f"shift of {r}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(1, 48, 32), (5, 40, 24), (8, 1024, 256), (3, 4096, 512), (17, 130, 96), (64, 256, 4096), (90, 256, 128),
                                   (70, 52, 40), (513, 1024, 320), (300, 300, 64), (2000, 512, 192), (129, 6144, 4096),
                                   (40, 5120, 4096), (1100, 2560, 64)])
def test_products_that_pass_a_gate(ops, sizes, dtype):
    """``x += scale sigmoid(gate + bias) (a w^T)`` for the sizes that every form of the product takes."""
    from tinyinfer_b200.parts.base import GatedSum
    t, n, k = sizes
    g = torch.Generator().manual_seed(t + n)
    a = torch.randn((t, k), generator=g).to(dtype)
    w = (torch.randn((n, k), generator=g) / k ** 0.5).to(torch.bfloat16)
    gate, bias, x = torch.randn((t, n + 12), generator=g) * 2, torch.randn((n,), generator=g), torch.randn((t, n), generator=g)
    y = a.double() @ w.double().T
    add = -0.7 * torch.sigmoid(gate[:, 4:4 + n].double() + bias.double()) * y
    d = x.to(DEV)
    ops.linear(a.to(DEV), w.to(DEV), GatedSum(d, gate.to(DEV)[:, 4:4 + n], bias.to(DEV), -0.7), accumulate=True, may_defer=True)
    ops.flush()
    ops.check_status()
    _close(d - x.to(DEV), add, torch.float32 if dtype == torch.float32 else torch.bfloat16, "through the product")
    assert (d.cpu().double() - (x.double() + add)).abs().max() < 1e-4 * add.abs().max() + 1e-5      # operands are exact here
    # a result that is there already
    d = x.to(DEV)
    ops.gated_add(y.float().to(DEV), GatedSum(d, gate.to(DEV)[:, 4:4 + n], bias.to(DEV), -0.7))
    _close(d - x.to(DEV), add, torch.float32, "added")


@pytest.mark.parametrize("sizes", [(1, 64, 48, 40), (8, 1024, 3072, 1024), (3, 96, 64, 2080), (16, 2048, 48, 2048), (33, 128, 512, 256),
                                   (64, 40, 40, 64), (8, 72, 16, 96)])
def test_two_products_of_few_rows_in_one_launch(ops, sizes):
    """A product that waits for the next one gives the same bits as by itself, beside a plain product and
    beside one whose epilogue is a gated activation; what cannot share a launch is launched by itself."""
    t, n1, n2, k = sizes
    g = torch.Generator().manual_seed(n1)
    rand = lambda *s: (torch.randn(s, generator=g) / s[-1] ** 0.5).to(torch.bfloat16).to(DEV)
    a1, a2, w1, w2 = rand(t, k), rand(t, k), rand(n1, k), rand(n2, k)
    gate_up, down = ops.pack_gate_up(rand(n2, k), rand(n2, k)), rand(k, n2)
    empty = lambda n: torch.full((t, n), float("nan"), dtype=torch.float32, device=DEV)

    def both(pair):
        ops.pair_few_rows = pair
        before, outs = ops.launches, [empty(n1), empty(n2), empty(n1), torch.zeros((t, k), device=DEV), empty(n1), empty(n2)]
        ops.linear(a1, w1, outs[0], may_pair=True)
        ops.linear(a2, w2, outs[1])
        ops.linear(a1, w1, outs[2], may_pair=True)
        ops.glu_ffn(a2, gate_up, down, outs[3], "gelu_tanh", 0.0, 0.0)
        count = ops.launches - before
        ops.linear(a1, w1, outs[4], may_pair=True)
        ops.linear(a1[:, :32].contiguous(), w2[:, :32].contiguous(), outs[5])          # another k
        ops.linear(a1, w1, outs[0], may_pair=True)
        ops.flush()
        return outs, count

    try:
        (apart, more), (together, fewer) = both(False), both(True)
    finally:
        ops.pair_few_rows = True
    assert fewer < more or k % 32 != 0
    for x, y in zip(apart, together):
        assert torch.equal(x, y)
    want = a2.double() @ w2.double().T
    _close(together[1], want.cpu(), torch.bfloat16, "second product")


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_time_convolution_with_biases(ops, taps):
    """A bias on the inputs (zeros, not the bias, lie before a sequence's start) and one on the result."""
    c = 40
    g = torch.Generator().manual_seed(taps)
    x = {r: torch.randn((n, c + 6), generator=g) for r, n in COUNTS.items()}
    w, b_in, b_out = torch.randn((c, taps), generator=g), torch.randn((c,), generator=g), torch.randn((c,), generator=g)
    state = _state(5 + (taps - 1) * c)
    got = {r: [] for r in COUNTS}

    def run(cut, at, step):
        rows = torch.cat([x[r][at[r]:at[r] + n] for r, n in cut]).to(DEV)
        out = torch.empty((rows.shape[0], c), dtype=torch.float32, device=DEV)
        ops.causal_conv(rows[:, 3:3 + c], w.to(DEV), step, state, 5, out, renew=True, in_bias=b_in.to(DEV), bias=b_out.to(DEV))
        o = 0
        for r, n in cut:
            got[r].append(out[o:o + n].cpu())
            o += n

    _walk(state, run)
    for r in COUNTS:
        want = plain.time_conv(x[r][:, 3:3 + c].double() + b_in.double(), w.double(), b_out.double())
        assert (torch.cat(got[r]).double() - want).abs().max() < 1e-5, r
    assert state.state[:, :5].abs().max() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(1, 48, 40), (9, 36, 31), (70, 128, 192), (300, 64, 96), (3, 40, 24), (5, 64, 96), (40, 128, 64),
                                   (150, 72, 33)])
def test_gelu_feed_forward(ops, sizes, dtype):
    from tinyinfer_b200.config.plan import PartSpec
    t, width, ff = sizes
    g = torch.Generator().manual_seed(ff)
    w = mlp_weights(ff, width, g)
    h = (torch.randn((t, width), generator=g) * 1.5).to(dtype)
    part = _part(ops, "ffn", PartSpec("glu_mlp", {"hidden_size": width, "intermediate_size": ff, "activation": "gelu_tanh"}), w)
    res = torch.zeros((t, width), dtype=torch.float32, device=DEV)
    part.forward(ops, h.to(DEV), res, None)
    _close(res, plain.mlp({k: v.double() for k, v in w.items()}, "", h.double()), dtype, "feed-forward")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("geom", [(4, 2, 12, 8, 6, 8), (1, 1, 16, 16, 16, 16), (6, 3, 10, 24, 0, 16), (8, 1, 80, 64, 40, 16)])
@pytest.mark.parametrize("share", [None, 0.3, -0.2, 1.0])
def test_row_norm_half_turn_and_mixed_values(ops, geom, share, dtype):
    from tinyinfer_b200.parts.rope import NoPosition, RopeNeox
    heads, kv, dk, dv, rot, ps = geom
    ctx, ql = [37, 5, 300], [9, 5, 1]
    step, cache, bt, positions, req = _paged(ctx, ql, ps, kv * (dk + dv), dtype)
    g = torch.Generator().manual_seed(3)
    t = len(positions)
    nq, nk, nv = heads * dk, kv * dk, kv * dv
    proj = torch.randn((t, nq + nk + nv + 5), generator=g) * torch.logspace(-1, 1, nq + nk + nv + 5)[None]
    qw, kw = 1 + 0.3 * torch.randn((nq,), generator=g), 1 + 0.3 * torch.randn((nk,), generator=g)
    first = torch.randn((t, nv + 3), generator=g) * 3
    rotation = (RopeNeox(dk, 777.0, rot) if rot else NoPosition()).rotation(DEV)
    q_out = torch.empty((t, nq), dtype=dtype, device=DEV)
    ops.qkv_turn_store(proj.to(DEV), rotation, None, step, cache, q_out, heads, kv, dk, dv,
                       row_norm=(qw.to(DEV), kw.to(DEV), 1e-5),
                       value_mix=None if share is None else (first.to(DEV)[:, 2:2 + nv], share))
    p64, pos = proj.double(), torch.tensor(positions)
    freq = plain.frequencies(777.0, rot)
    q_want = plain.turn_halves((plain.unit_rms(p64[:, :nq], 1e-5) * qw.double()).view(t, heads, dk), pos, freq)
    k_want = plain.turn_halves((plain.unit_rms(p64[:, nq:nq + nk], 1e-5) * kw.double()).view(t, kv, dk), pos, freq)
    v_want = p64[:, nq + nk:nq + nk + nv]
    if share is not None:
        v_want = (1 - share) * v_want + share * first[:, 2:2 + nv].double()
    v_want = v_want.view(t, kv, dv)
    _close(q_out.view(t, heads, dk), q_want, dtype, "queries")
    for i in range(t):
        page = cache.pages[int(bt[req[i], positions[i] // ps])]
        slot = positions[i] % ps
        _close(page[: kv * ps * dk].view(kv, ps, dk)[:, slot], k_want[i], dtype, f"key of token {i}")
        _close(page[kv * ps * dk:].view(kv, ps, dv)[:, slot], v_want[i], dtype, f"value of token {i}")


@pytest.mark.parametrize("sizes", [(1, 5, 3, 16.0), (40, 130, 16, 4.0), (17, 64, 70, 1.0), (300, 96, 33, 9.5)])
def test_decay_of_the_key_channels(ops, sizes):
    t, n, rank, tau = sizes
    g = torch.Generator().manual_seed(n)
    wide = torch.randn((t, rank + 7), generator=g) * 2
    bias = torch.randn((n,), generator=g) * 3
    for a2 in (torch.randn((n, rank), generator=g), torch.randn((n, rank), generator=g).to(torch.bfloat16)):
        out = torch.empty((t, n), dtype=torch.float32, device=DEV)
        ops.low_rank_decay(wide.to(DEV)[:, 4:4 + rank], a2.to(DEV), bias.to(DEV), tau, out)
        want = torch.sigmoid(wide[:, 4:4 + rank].double() @ a2.double().T + bias.double()) ** (1.0 / tau)
        assert (out.cpu().double() - want).abs().max() < 1e-5


# ---- the recurrence per channel ------------------------------------------------------------------------
def _gates(ops, blocks, per, g, dtype=torch.bfloat16):
    wr, wi = ((torch.randn((blocks, per, per), generator=g) * 2 / per ** 0.5).to(dtype) for _ in range(2))
    return wr, wi, ops.pack_block_gates(wr.to(DEV), wi.to(DEV))


def _plain_recurrence(u, y, wr, wi, gate_bias, log_decay, y_bias, s=None):
    blocks = wr.shape[0]
    r = torch.sigmoid(plain.block_diagonal(u, wr, gate_bias[0].view(blocks, -1)))
    i = torch.sigmoid(plain.block_diagonal(u, wi, gate_bias[1].view(blocks, -1)))
    log_a = log_decay * r
    s = torch.zeros_like(u[0]) if s is None else s
    rows = []
    for t in range(u.shape[0]):
        s = torch.exp(log_a[t]) * s + torch.sqrt(1.0 - torch.exp(2.0 * log_a[t])) * i[t] * u[t]
        rows.append(s)
    return torch.stack(rows) * plain.gelu_tanh(y + y_bias), s


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("geom", [(1, 7), (3, 20), (2, 64), (5, 33), (4, 256), (1, 800), (40, 4)])
def test_gated_recurrence_through_all_its_forms(ops, geom, dtype):
    """Portions long and short, single tokens, and steps of many rows pass the state to one another; more
    requests than a block takes; slots in another order than the requests."""
    blocks, per = geom
    n = blocks * per
    g = torch.Generator().manual_seed(n)
    wr, wi, gates = _gates(ops, blocks, per, g)
    gate_bias, y_bias = torch.randn((2, n), generator=g), torch.randn((n,), generator=g)
    log_decay = -torch.exp(torch.randn((n,), generator=g) * 1.5 - 2)
    names = [f"r{i}" for i in range(19)]
    cuts = [[("r0", 130), ("r1", 3)], [(r, 1) for r in names], [("r1", 57), ("r0", 56), ("r2", 2), ("r3", 1)],
            [(r, 1) for r in names[::-1]], [("r4", 1)], [("r5", 7), ("r0", 1)]]
    total = {r: sum(c for cut in cuts for q, c in cut if q == r) for r in names}
    u = {r: torch.randn((c, n), generator=g) for r, c in total.items()}
    y = {r: torch.randn((c, n), generator=g) for r, c in total.items()}
    slot = {r: (7 * i + 3) % 19 for i, r in enumerate(names)}
    state = _state(n + 5, slots=19)
    at, got = {r: 0 for r in names}, {r: [] for r in names}
    for cut in cuts:
        step, state.slots = _rows_step([c for _, c in cut], [slot[r] for r, _ in cut])
        rows = lambda src: torch.cat([src[r][at[r]:at[r] + c] for r, c in cut]).to(DEV)
        wide = torch.cat([rows(y), torch.zeros((len(rows(y)), 3), device=DEV)], dim=1)
        out = torch.empty((wide.shape[0], n), dtype=dtype, device=DEV)
        ops.gated_recurrence(rows(u), gates, gate_bias.to(DEV), log_decay.to(DEV), wide[:, :n], y_bias.to(DEV), step, state, out)
        o = 0
        for r, c in cut:
            got[r].append(out[o:o + c].cpu())
            at[r] += c
            o += c
    ops.check_status()
    d = lambda x: x.double()
    for r in names:
        want, last = _plain_recurrence(d(u[r]), d(y[r]), d(wr), d(wi), d(gate_bias), d(log_decay), d(y_bias))
        _close(torch.cat(got[r]), want, dtype, f"rows of {r}")
        # the state itself is float32 in both engines
        assert (state.state[slot[r], :n].cpu().double() - last).abs().max() < 3e-5 * max(1.0, float(last.abs().max())), r
    assert state.state[:, n:].abs().max() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decoded", [False, True])
def test_an_early_input_is_still_there_hundreds_of_tokens_later(ops, decoded, dtype):
    """Only the first token has an input; afterwards the state shrinks by a known factor per token."""
    blocks, per, t = 2, 16, 650
    n = blocks * per
    g = torch.Generator().manual_seed(0)
    _, _, gates = _gates(ops, blocks, per, g)
    zero = ops.pack_block_gates(torch.zeros_like(gates.rows[:, :per]), torch.zeros_like(gates.rows[:, per:]))
    rate = torch.linspace(0.0, 0.01, n)                       # log a = -rate: r = sigmoid(0) = 1/2
    u = torch.zeros((t, n))
    u[0] = torch.randn((n,), generator=g)
    y = torch.full((t, n), 12.0)                              # gelu(12) = 12
    gate_bias = torch.cat([torch.zeros((1, n)), torch.full((1, n), 40.0)])
    state, at = _state(n), 0
    for c in ([300, 2, 300] + [1] * 48 if decoded else [129, 2, 519]):
        step, state.slots = _rows_step([c], [1])
        out = torch.empty((c, n), dtype=dtype, device=DEV)
        ops.gated_recurrence(u[at:at + c].contiguous().to(DEV), zero, gate_bias.to(DEV), (-2 * rate).to(DEV),
                             y[at:at + c].contiguous().to(DEV), torch.zeros((n,), device=DEV), step, state, out)
        at += c
    assert at == t
    r64 = rate.double()
    want = torch.sqrt(-torch.expm1(-2 * r64)) * u[0].double() * torch.exp(-r64 * (t - 1))
    assert (state.state[1].cpu().double() - want).abs().max() < 2e-6
    assert (out[-1].cpu().double() / 12.0 - want).abs().max() < (2e-6 if dtype == torch.float32 else 1e-2)
    assert state.state[0].abs().max() == 0 and state.state[2].abs().max() == 0


@pytest.mark.parametrize("decoded", [False, True])
def test_a_far_write_is_read_back(ops, decoded):
    """Token 0 writes a one-hot value under a key channel of its own; 700 tokens with other keys follow; the last
    token asks for the first key.  A channel that forgets nothing gives it back whole, one that forgets at a
    known rate shows it against the norm's eps."""
    heads, dk, dv, t, eps = 2, 16, 8, 701, 1e-6
    g = torch.Generator().manual_seed(1)
    k = torch.zeros((t, heads, dk))
    for h in range(heads):
        k[torch.arange(1, t), h, 1 + torch.arange(1, t) % (dk - 1)] = 3.0      # never the first channel again
    k[0, :, 0] = 5.0
    q = k.clone()
    q[-1] = 0
    q[-1, :, 0] = 8.0
    v = torch.randn((t, heads, dv), generator=g)
    v[0] = 0
    v[0, 0, 3] = v[0, 1, 5] = 1.0
    ones = torch.ones((dv,), device=DEV)
    for rate in (0.0, 0.005):
        decay = torch.rand((t, heads, dk), generator=g)
        decay[:, :, 0] = math.exp(-rate)
        state, at = _state(heads * dk * dv), 0
        for n in ([300, 2, 348] + [1] * 51 if decoded else [129, 2, 570]):
            step, state.slots = _rows_step([n], [1])
            out = torch.empty((n, heads * dv), dtype=torch.float32, device=DEV)
            dev = lambda x: x[at:at + n].reshape(n, -1).contiguous().to(DEV)
            ops.matrix_state("decayed_sum", dev(q), dev(k), dev(v), None, None, None, None, step, state, out, heads=heads,
                             kv_heads=heads, dk=dk, dv=dv, eps=eps, norm_weight=ones, decay=dev(decay))
            at, last = at + n, out[-1].cpu().double().view(heads, dv)
        assert at == t
        o = 8.0 * dk ** -0.5 * 5.0 * math.exp(-rate * (t - 1))
        want = o / math.sqrt(o * o / dv + eps)
        for head, col in ((0, 3), (1, 5)):
            assert abs(float(last[head, col]) - want) < 2e-4 * max(1.0, want), (rate, last[head], want)
            rest = last[head].clone()
            rest[col] = 0
            assert rest.abs().max() < 1e-4
    assert state.state[0].abs().max() == 0 and state.state[2].abs().max() == 0


# ---- parts alone ---------------------------------------------------------------------------------
def _part(ops, category, spec, w):
    from tinyinfer_b200.parts.base import build_part
    part = build_part(category, spec)
    part.load_weights({k: v.to(DEV) for k, v in w.items()}, ops)
    return part


def _mixer_part(ops, entry, width, w, value_mix=None):
    from tinyinfer_b200.config import vametar
    cfg = SimpleNamespace(width=width, norm_eps=1e-5)
    layer = vametar.VametarLayer(entry["type"], vametar._mixer(entry, "here", entry["type"]), None)
    return _part(ops, "mixer", vametar._mixer_spec(cfg, layer, value_mix), w)


def _plain_mixer(entry, w, x):
    w64 = {k: v.double() for k, v in w.items()}
    if entry["type"] == "attention":
        return plain.attention(w64, "", x, entry["mixer"], 1e-5)[0]
    return plain.rglru(w64, "", x, entry["mixer"]) if entry["type"] == "rglru" else plain.gla(w64, "", x, entry["mixer"], 1e-5)


MIXER_CASES = [attention(4, 2, 12, 8, 6, 1000.0, 0.29), attention(1, 1, 16, 16, 0, 7.0, 0.25), attention(3, 3, 8, 8, 2, 30.0, 0.35),
               attention(4, 2, 64, 64, 32, 20000.0, 0.125), attention(2, 1, 128, 128, 128, 300000.0, 0.09),
               attention(6, 6, 80, 32, 40, 250.0, 0.1), attention(6, 2, 32, 16, 32, 900.0, 0.18),
               rglru(60, 3, 3), rglru(36, 1, 1), rglru(8, 8, 6), rglru(192, 3, 4), rglru(128, 8, 2), rglru(35, 5, 16),
               gla(3, 8, 20, 9.0), gla(1, 16, 16, 1.0), gla(2, 64, 192, 16.0), gla(4, 128, 32, 5.0), gla(1, 200, 96, 2.0),
               gla(5, 3, 7, 12.0), gla(2, 256, 64, 4.0)]
CUTS = [[("a", 30), ("b", 1)], [("b", 2), ("c", 5)], [("a", 1), ("b", 30), ("c", 1)], [("a", 2), ("c", 1)],
        [("a", 17), ("b", 7), ("c", 33)], [("a", 1)], [("a", 1), ("c", 2)], [("b", 0), ("d", 70)], [("d", 1), ("a", 1)]]
TOTAL = {"a": 53, "b": 40, "c": 42, "d": 71}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("entry", MIXER_CASES, ids=lambda e: e["type"] + "-" + "-".join(str(v) for v in e["mixer"].values() if not isinstance(v, dict)))
def test_each_mixer_alone_in_portions(ops, entry, dtype):
    """Four requests in portions down to one token; the fourth takes the slot that the second gave back."""
    width = 64
    g = torch.Generator().manual_seed(5)
    w = mixer_weights(entry["type"], entry["mixer"], width, g, v_mix=False)
    part = _mixer_part(ops, entry, width, w)
    inputs = {r: torch.randn((n, width), generator=g).to(dtype).float() for r, n in TOTAL.items()}
    got = _run_mixer(ops, part, inputs, CUTS, dtype)
    for r, x in inputs.items():
        _close(got[r], _plain_mixer(entry, w, x.double()), dtype, f"{entry['type']} request {r}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("entry", [gla(2, 64, 64, 16.0), gla(1, 32, 128, 2.0), gla(2, 128, 160, 7.0), rglru(96, 2, 4), rglru(40, 5, 3)],
                         ids=lambda e: e["type"] + str(next(iter(e["mixer"].values()))))
def test_recurrences_over_long_portions(ops, entry, dtype):
    """Portions long enough that a head's state columns are cut over several blocks, between portions that
    are not; a slot that a finished request gave back starts at zero again."""
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


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decoded", [False, True])
def test_one_key_stands_out(ops, decoded, dtype):
    """A layer whose query at the last token points at one key alone, which carries a value of its own: the
    first tokens, both sides of page borders, hundreds of positions back, the query's own, and (in a portion)
    the token right after the query, which must not be seen."""
    width, dim, ps = 64, 24, 16
    entry = attention(2, 1, dim, 8, 4, 100.0, 1.0)
    w = {"q": torch.zeros((2 * dim, width)), "k": torch.zeros((dim, width)), "v": torch.zeros((8, width)),
         "q.norm": torch.full((2 * dim,), 3.0), "k.norm": torch.full((dim,), 3.0), "o": torch.zeros((width, 16))}
    for a in range(2):                                          # rows 4 .. 23 of a head are not turned
        w["q"][a * dim + 4:(a + 1) * dim, :20] = torch.eye(20)
    w["k"][4:, :20] = torch.eye(20)
    w["v"][:, 40:48] = torch.eye(8)
    w["o"][:16, :] = torch.eye(16)
    part = _mixer_part(ops, entry, width, {k: v.to(torch.bfloat16) for k, v in w.items()})
    for pos, targets in ((700, [0, 1, 15, 16, 17, 351, 352, 687, 688, 699, 700]), (16, [0, 15, 16]), (1, [0, 1])):
        for target in targets:
            g = torch.Generator().manual_seed(target)
            x = torch.zeros((pos + 2, width))
            x[:, :20] = torch.nn.functional.normalize(torch.randn((pos + 2, 20), generator=g), dim=1)
            direction = torch.nn.functional.normalize(torch.randn((20,), generator=g), dim=0)
            x[:, :20] -= 0.9 * (x[:, :20] @ direction).clamp(min=0)[:, None] * direction         # no other key comes near
            x[target, :20] = x[pos, :20] = direction
            x[pos + 1, :20] = direction                          # right after the query
            x[:, 41] = 1.0
            x[target, 40], x[target, 41] = 1.0, 0.0
            x = x.to(dtype).float()
            cuts = [[("a", pos)], [("a", 1)], [("a", 1)]] if decoded else [[("a", max(1, pos - 40))], [("a", pos + 2 - max(1, pos - 40))]]
            row = _run_mixer(ops, part, {"a": x}, cuts, dtype, page_size=ps)["a"][pos]
            # the query's own key has the same direction as the target's: the two share the weight
            share = 1.0 if target == pos else 0.5
            got = torch.stack([row[0], row[8]])
            assert ((got - share).abs() < 0.03).all(), f"query {pos}, key {target}: {got.tolist()}"


def test_the_gate_and_the_shift_of_a_layer(ops):
    """The block around a mixer that adds its result by other means than one closing product: the same sum."""
    from tinyinfer_b200.parts.base import Part
    from tinyinfer_b200.parts.block import GatedPreNormBlock
    from tinyinfer_b200.parts.norm import RMSNorm
    width, t = 40, 11
    g = torch.Generator().manual_seed(6)
    w = {"shift": torch.randn((width,), generator=g) * 0.5, "rg1": torch.randn((width, width), generator=g) / width ** 0.5,
         "rg1.b": torch.randn((width,), generator=g)}
    norm_w = torch.tensor(1.3)

    class Doubled(Part):
        def __init__(self, closing):
            self.ends_in_linear = closing

        def cache_spec(self):
            return None

        def forward(self, ops, h, residual, step, cache):
            two = torch.eye(width, device=DEV) * 2
            if self.ends_in_linear:
                ops.linear(h, two, residual, accumulate=True)
            else:
                residual += 2 * h.float()

    x = torch.randn((t, width), generator=g)
    w64 = {k: v.double() for k, v in w.items()}
    h = plain.scalar_norm(x.double(), norm_w.double(), 1e-5)
    want = x.double() - 0.6 * plain.gated(w64, "rg1", h, 2 * plain.token_shift(h, w64["shift"]))
    for closing in (False, True):
        norm = RMSNorm(width, 1e-5, scalar=True)
        norm.load_weights({"weight": norm_w.to(DEV)}, ops)
        block = GatedPreNormBlock(Doubled(closing), norm, hidden_size=width, multiplier=-0.6)
        block.load_weights({k: v.to(DEV) for k, v in w.items()}, ops)
        state = _state(width)
        step, state.slots = _rows_step([t], [1])
        step.act_dtype = torch.float32
        d = x.to(DEV)
        cache = type("C", (), {"__getitem__": lambda s, n: state, "child": lambda s, n: None})()
        block.forward(ops, d, step, cache)
        _close(d, want, torch.float32, f"closing product: {closing}")
        _close(state.state[1], h[-1], torch.float32, "kept row")


# ---- whole models ---------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
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
    ("C", "long portions", "bfloat16"), ("C", "long portions", "float32"), ("D", "mixed", "float32"), ("D", "tail", "bfloat16")])
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


@pytest.mark.parametrize("seed", range(16))
def test_drawn_configurations(tmp_path_factory, seed):
    """Sizes, constants, options and the order of layers drawn from a seed: mixed batches in a small pool in
    float32, whole prompts in bfloat16."""
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


def test_float32_cuttings_give_the_same_bits(tmp_path_factory):
    d = make_model(tmp_path_factory.getbasetemp(), "A")
    reqs = _requests("A")
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
            assert err.max() < 5e-2, f"{r}: {float(err.max())}"
    assert all(n == 24 for n in eng.cache.free_pages())


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["A", "B", "D"])
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
        if entry["type"] == "gla":                       # no stored tensor says it
            entry["mixer"]["decay_rank"] = 24
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
