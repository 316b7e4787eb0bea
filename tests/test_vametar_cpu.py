"""Vametar without a GPU: its configuration and plan, what a request keeps, and the plain
implementation's mechanisms at their edges."""
import copy
import math

import pytest
import torch

import plain_vametar as plain
from tinyinfer_b200.cache import CacheManager
from tinyinfer_b200.config import ConfigError, VametarConfig, architecture_of, known_architectures
from tinyinfer_b200.config.vametar import build_plan
from tinyinfer_b200.parts.base import CompositeSpec, FixedStateSpec, PagedKVSpec
from tinyinfer_b200.parts.model import CausalLM
from tinyinfer_b200.weights.loader import check_tensors
from util import random_tokens
from vametar_util import SMALL, SMALL_A, SMALL_B, SMALL_C, SMALL_D, drawn_configuration, random_weights

F = torch.float64


def _plan(cfg):
    return build_plan(VametarConfig.from_dict(cfg))


def test_the_registry_chooses_it():
    assert "Vametar" in known_architectures() and "vametar" in known_architectures()
    assert architecture_of(SMALL_A).name == "Vametar"
    assert VametarConfig.from_dict(SMALL_A).to_dict() == SMALL_A


@pytest.mark.parametrize("path, value, message", [
    ("vocab", None, "lacks 'vocab'"), ("width", 0, "'width' must be >= 1"), ("norm.eps", 0.0, "'norm.eps'"),
    ("residual_mult", None, "lacks 'residual_mult'"), ("residual_mult", "1", "'residual_mult'"),
    ("logit_scale", None, "lacks 'logit_scale'"), ("embedding.bigram", None, "lacks 'embedding.bigram.buckets'"),
    ("embedding.bigram.buckets", 0, "'embedding.bigram.buckets'"), ("embedding.bigram.mul_prev", 1.5, "mul_prev"),
    ("layers", [], "'layers'"), ("layers.0.type", "conv", "'layers[0].type' is 'conv'"),
    ("layers.0.mixer", None, "'layers[0].mixer'"), ("layers.0.mixer.blocks", 7, "does not fall into 7"),
    ("layers.0.mixer.conv", 0, "'mixer.conv'"), ("layers.0.mlp.kind", "moe", "'layers[0].mlp.kind'"),
    ("layers.0.mlp.ff", None, "lacks 'ff'"), ("layers.1.mixer.kv_heads", 3, "4 heads cannot share 3"),
    ("layers.1.mixer.rot.dims", 14, "rot.dims"), ("layers.1.mixer.rot.dims", 5, "rot.dims"),
    ("layers.1.mixer.scale", None, "lacks 'mixer.scale'"), ("layers.2.mixer.tau", -1.0, "'mixer.tau'"),
    ("layers.4.mixer.vdim", 10, "cannot be mixed with the 16 elements of layer 1")])
def test_configuration_errors(path, value, message):
    cfg = copy.deepcopy(SMALL_A)
    node = cfg
    keys = [int(k) if k.isdigit() else k for k in path.split(".")]
    for k in keys[:-1]:
        node = node[k]
    node[keys[-1]] = value
    with pytest.raises(ConfigError) as e:
        VametarConfig.from_dict(cfg)
    assert message in str(e.value)


@pytest.mark.parametrize("cfg", [*SMALL.values(), *(drawn_configuration(s) for s in range(30))])
def test_tensor_names_and_shapes(cfg):
    want = CausalLM(_plan(cfg)).expected_tensors()
    have = {k: tuple(v.shape) for k, v in random_weights(cfg, 0).items()}
    assert set(want) == set(have)
    check_tensors("here", want, have)


def test_the_first_layer_that_mixes_values_is_their_source():
    roles = [lp.mixer.params.get("value_mix") for lp in _plan(SMALL_A).layers]
    assert roles == [None, "source", None, None, "mix", None, "mix"]
    assert [lp.mixer.params.get("value_mix") for lp in _plan(SMALL_B).layers] == ["source", None, None, None, None]
    # the source's own share may be missing from a folder, a later layer's may not
    want = CausalLM(_plan(SMALL_A)).expected_tensors()
    assert want["l1.mix.vmix"].optional and not want["l4.mix.vmix"].optional and "l3.mix.vmix" not in want


def test_what_a_request_keeps():
    model = CausalLM(_plan(SMALL_A))
    specs = model.cache_specs()
    assert len(specs) == 8 and model.embedding_slot == 7 and specs[7] == FixedStateSpec((1,), torch.int32)
    assert model.cache_keys() == [(i, True) for i in range(8)]
    assert all(isinstance(s, CompositeSpec) and dict(s.flat())["shift"] == FixedStateSpec((48,), torch.float32)
               for s in specs[:7])
    kept = [dict(s.flat())["mixer"] for s in specs[:7]]
    assert kept[0] == FixedStateSpec((60 * 3,), torch.float32)          # the state and two rows of the convolution
    assert kept[1] == PagedKVSpec(2, 12, None, 8, 0, None)
    assert kept[2] == FixedStateSpec((3 * 8 * 20,), torch.float32)
    assert dict(CausalLM(_plan(SMALL_B)).cache_specs()[1].flat())["mixer"] == FixedStateSpec((36,), torch.float32)


def test_state_slots_without_pages_and_used_again():
    cm = CacheManager(CausalLM(_plan(SMALL_D)).cache_specs(), page_size=8, num_pages=1, max_requests=2, device="cpu")
    assert cm.groups == []
    cm.reserve_step([("a", 1000), ("b", 1)])                    # no attention: a request may be longer than the pool
    slots = torch.tensor([cm.state_slot("a"), cm.state_slot("b")], dtype=torch.int32)
    token = cm.view(2, True, [], slots)
    assert token.state.dtype == torch.int32 and token.state.shape == (3, 1)
    token.state[cm.state_slot("a")] = 9
    row = cm.view(0, True, [], slots)["shift"].state
    row[cm.state_slot("a")] = 1.0
    was = cm.state_slot("a")
    cm.free_request("a")
    cm.reserve_step([("c", 2)])
    assert cm.state_slot("c") == was and int(token.state[was]) == 0 and float(row[was].abs().max()) == 0.0
    cm.check()


# ---- the plain mechanisms at their edges ---------------------------------------------------------------
def test_plain_hash_of_two_tokens():
    assert plain.bigram_rows([5, 7, 7, 0], 10, 3, 13) == [13, (50 + 21) % 13, (70 + 21) % 13, 70 % 13]
    assert plain.bigram_rows([5], 10, 3, 13) == [13]
    assert plain.bigram_rows([1, 2, 3], 4, 4, 1) == [1, 0, 0]
    cfg = {"embedding": {"bigram": {"buckets": 2, "mul_prev": 1, "mul_cur": 0}}}
    w = {"embed": torch.tensor([[1.0], [2.0]], dtype=F), "bigram": torch.tensor([[10.0], [20.0], [30.0]], dtype=F)}
    assert plain.embed(cfg, w, [1, 0, 1]).view(-1).tolist() == [32.0, 21.0, 12.0]


def test_plain_shift_gelu_and_convolution():
    h = torch.tensor([[1.0, 10.0], [2.0, 20.0], [4.0, 40.0]], dtype=F)
    mu = torch.tensor([1.0, 0.5], dtype=F)
    assert plain.token_shift(h, mu).tolist() == [[0.0, 5.0], [1.0, 15.0], [2.0, 30.0]]
    z = torch.tensor([0.0, 30.0, -30.0, 1.0], dtype=F)
    assert torch.allclose(plain.gelu_tanh(z), torch.tensor([0.0, 30.0, 0.0, 0.5 * (1 + math.tanh(
        math.sqrt(2 / math.pi) * 1.044715))], dtype=F), atol=1e-12)
    u = torch.arange(1.0, 5.0, dtype=F).view(4, 1)
    y = plain.time_conv(u, torch.tensor([[100.0, 10.0, 1.0]], dtype=F), torch.tensor([0.5], dtype=F))
    assert y.view(-1).tolist() == [1.5, 12.5, 123.5, 234.5]
    mats = torch.tensor([[[0.0, 1.0], [1.0, 0.0]], [[2.0, 0.0], [0.0, 3.0]]], dtype=F)
    bias = torch.tensor([[0.0, 0.1], [0.2, 0.3]], dtype=F)
    got = plain.block_diagonal(torch.tensor([[1.0, 2.0, 3.0, 4.0]], dtype=F), mats, bias)
    assert torch.allclose(got, torch.tensor([[2.0, 1.1, 6.2, 12.3]], dtype=F))


def test_plain_recurrences_by_hand():
    one, zero = torch.ones((1, 1), dtype=F), torch.zeros((1,), dtype=F)
    w = {"x": one, "x.b": zero, "y": one * 0, "y.b": zero + 30.0, "conv": one, "conv.b": zero, "ra": one[None] * 0,
         "ra.b": zero[None], "ri": one[None] * 0, "ri.b": zero[None] + 40.0, "lam": zero, "o": one / 30.0}
    m = {"width": 1, "blocks": 1, "conv": 1}
    # r = 1/2, i = 1, log a = -4 ln 2: a = 1/16, and the branch in front of the output is 30
    out = plain.rglru(w, "", torch.tensor([[1.0], [0.0], [2.0]], dtype=F), m).view(-1)
    b = math.sqrt(1 - 1 / 256)
    assert torch.allclose(out, torch.tensor([b, b / 16, b / 256 + 2 * b], dtype=F))
    # a key channel that never forgets beside one that halves: alpha = 1/2 for z = 0 and tau = 1
    eye = torch.eye(2, dtype=F)
    g = {"q": eye * 2 ** 0.5, "k": eye, "v": eye, "g": eye * 0, "a1": eye * 0, "a2": eye, "a2.b": torch.tensor([60.0, 0.0], dtype=F),
         "norm": torch.ones(2, dtype=F), "o": eye}
    h = torch.tensor([[1.0, 0.0], [0.0, 1.0], [1.0, 1.0]], dtype=F)
    # S before the read of token 2: e0 e0^T + 1/2 e1 e1^T + (1,1)(1,1)^T; the norm leaves directions, the gate is silu(0) = 0
    assert plain.gla(g, "", h, {"heads": 1, "dim": 2, "vdim": 2, "tau": 1.0}, 1e-9).abs().max() == 0
    g["g"] = torch.full((2, 2), 50.0, dtype=F)
    out = plain.gla(g, "", h, {"heads": 1, "dim": 2, "vdim": 2, "tau": 1.0}, 0.0)
    read = torch.tensor([3.0, 2.5], dtype=F)
    assert torch.allclose(out[2], read / read.pow(2).mean().sqrt() * 100.0)


def test_plain_values_are_mixed_with_the_first_layers():
    cfg = copy.deepcopy(SMALL_A)
    w = {k: v.to(F) for k, v in random_weights(cfg, 3).items()}
    tokens = random_tokens(cfg["vocab"], 9, seed=1)
    base = plain.forward(cfg, w, tokens)
    assert (base - plain.forward(cfg, {**w, "l1.mix.vmix": w["l1.mix.vmix"] + 1}, tokens)).abs().max() == 0   # unused
    for name in ("l4.mix.vmix", "l6.mix.vmix"):
        assert (base - plain.forward(cfg, {**w, name: w[name] + 0.5}, tokens)).abs().max() > 1e-3
    # a share of 1 takes the source's values alone
    taken = {**w, "l4.mix.vmix": torch.tensor(1.0, dtype=F)}
    a = plain.forward(cfg, taken, tokens)
    assert (a - plain.forward(cfg, {**taken, "l4.mix.v": w["l4.mix.v"] * 0}, tokens)).abs().max() == 0


def test_plain_is_causal_and_greedy_continues_it():
    for cfg in (SMALL_A, SMALL_B, SMALL_C):
        w = {k: v.to(F) for k, v in random_weights(cfg, 1).items()}
        tokens = random_tokens(cfg["vocab"], 12, seed=2)
        rows = []
        whole = plain.forward(cfg, w, tokens, rows)
        assert len(rows) == len(cfg["layers"]) and rows[0].shape == (12, cfg["width"])
        for n in (1, 2, 7):
            assert torch.allclose(plain.forward(cfg, w, tokens[:n]), whole[:n], atol=1e-10)
        assert plain.greedy(cfg, w, tokens[:4], 2)[0] == int(whole[3].argmax())
