"""Saberax without a GPU: its configuration and plan, what a request keeps, positions, and the plain
implementation's mechanisms at their edges."""
import copy
import math

import pytest
import torch

import plain_saberax as plain
from saberax_util import SMALL, SMALL_A, SMALL_B, SMALL_C, drawn_configuration, random_weights
from tinyinfer_b200.cache import CacheManager
from tinyinfer_b200.config import ConfigError, SaberaxConfig, architecture_of, known_architectures
from tinyinfer_b200.config.saberax import build_plan
from tinyinfer_b200.parts.base import FixedStateSpec, PagedKVSpec
from tinyinfer_b200.parts.model import CausalLM
from tinyinfer_b200.parts.rope import RopeStretched, RopeWavelength
from tinyinfer_b200.weights.loader import check_tensors
from util import random_tokens

F = torch.float64


def _plan(cfg):
    return build_plan(SaberaxConfig.from_dict(cfg))


def test_the_registry_chooses_it():
    assert "Saberax" in known_architectures() and "saberax" in known_architectures()
    assert architecture_of(SMALL_A).name == "Saberax"
    assert SaberaxConfig.from_dict(SMALL_A).to_dict() == SMALL_A


@pytest.mark.parametrize("path, value, message", [
    ("vocab", None, "lacks 'vocab'"), ("width", 0, "'width' must be >= 1"), ("norm.eps", 0.0, "'norm.eps'"),
    ("residual_mult", None, "lacks 'residual_mult'"), ("residual_mult", "1", "'residual_mult'"),
    ("layers", [], "'layers'"), ("layers.0.type", "conv", "'layers[0].type' is 'conv'"),
    ("layers.0.mixer", None, "'layers[0].mixer'"), ("layers.0.mixer.left.mask", None, "lacks 'mixer.left.mask.size'"),
    ("layers.0.mixer.left.kv_heads", 3, "4 heads cannot share 3"), ("layers.0.mixer.left.rot.dims", 14, "rot.dims"),
    ("layers.0.mixer.left.rot.scaling.fast", None, "lacks 'mixer.left.rot.scaling.fast'"),
    ("layers.0.mixer.right.tau", -1.0, "'mixer.right.tau'"), ("layers.0.mlp.kind", "wide", "'layers[0].mlp.kind'"),
    ("layers.0.mlp.ff", None, "lacks 'ff'"), ("layers.1.mixer.vdim", 12, "the values are the keys of 10"),
    ("layers.1.mixer.rot.dims", 5, "rot.dims"), ("layers.1.mixer.rot.scaling.low", 0, "rot.scaling.low"),
    ("layers.1.mixer.mask.size", 0, "'mixer.mask.size'"), ("layers.1.mixer.scale", None, "lacks 'mixer.scale'"),
    ("layers.1.mlp.router.top", 9, "top 9 of 8"), ("layers.1.mlp.router.groups.count", 5, "12 experts do not fall into 5"),
    ("layers.1.mlp.router.groups.keep", 4, "of which 4"), ("layers.1.mlp.router.scale", None, "lacks 'router.scale'"),
    ("layers.1.mlp.shared.ff", None, "lacks 'shared.ff'"), ("layers.2.mixer.right.blocks", 7, "does not fall into 7"),
    ("layers.2.mixer.left.q_temp.every", 0, "q_temp.every"), ("layers.2.mixer.left.q_temp", None, "q_temp.coef"),
    ("layers.4.weights_of", 4, "must name another layer"), ("layers.4.weights_of", 9, "must name another layer"),
    ("layers.4.weights_of", 1, "differ"), ("layers.4.mixer.left.scale", 0.31, "differ"), ("layers.2.weights_of", 4, "leads back")])
def test_configuration_errors(path, value, message):
    cfg = copy.deepcopy(SMALL_A)
    node = cfg
    keys = [int(k) if k.isdigit() else k for k in path.split(".")]
    for k in keys[:-1]:
        node = node[k]
    node[keys[-1]] = value
    with pytest.raises(ConfigError) as e:
        SaberaxConfig.from_dict(cfg)
    assert message in str(e.value)


@pytest.mark.parametrize("cfg", [*SMALL.values(), *(drawn_configuration(s) for s in range(30))])
def test_tensor_names_and_shapes(cfg):
    want = CausalLM(_plan(cfg)).expected_tensors()
    have = {k: tuple(v.shape) for k, v in random_weights(cfg, 0).items()}
    assert set(want) == set(have)
    check_tensors("here", want, have)


def test_what_a_request_keeps():
    model = CausalLM(_plan(SMALL_A))
    specs = model.cache_specs()
    assert len(specs) == 6 and len(model.blocks) == 5
    assert dict(specs[0].flat()) == {"left": PagedKVSpec(2, 12, 21, 8, 0, None), "right": FixedStateSpec((3 * 8 * 20,), torch.float32)}
    assert specs[1] == PagedKVSpec(2, 10, None, None, 0, 19)
    assert dict(specs[2].flat()) == {"left": PagedKVSpec(3, 8, None, 12, 0, None), "right": FixedStateSpec((60 * 3,), torch.float32)}
    # the layer that runs a second time with the same tensors keeps things of its own
    assert specs[4] == specs[2] and [e.cache_slot for e in model.plan.schedule] == list(range(6))
    assert [e.layer for e in model.plan.schedule] == [0, 1, 2, 3, 2, 4]


def test_tensors_of_a_later_layer_and_of_a_layer_in_between():
    cfg = copy.deepcopy(SMALL_A)
    cfg["layers"].append(dict(cfg["layers"][2], weights_of=4))             # a chain
    cfg["layers"].insert(0, dict(cfg["layers"][3], weights_of=4))          # the owner comes behind
    for i in (5, 7):
        cfg["layers"][i] = dict(cfg["layers"][i], weights_of=cfg["layers"][i]["weights_of"] + 1)
    plan = _plan(cfg)
    assert [e.layer for e in plan.schedule] == [3, 0, 1, 2, 3, 2, 4, 2]
    assert plan.layers[3].names["mixer"] == "l4.mix." and plan.layers[2].names["mixer"] == "l3.mix."
    assert [plain.tensors_of(cfg, i) for i in range(8)] == [4, 1, 2, 3, 4, 3, 6, 3]


def test_pages_and_slots_used_again():
    cm = CacheManager(CausalLM(_plan(SMALL_A)).cache_specs(), page_size=8, num_pages=8, max_requests=2, device="cpu")
    cm.reserve_step([("a", 40), ("b", 10)])
    view = cm.view(0, True, [torch.zeros((2, 8), dtype=torch.int32)] * len(cm.groups),
                   torch.tensor([cm.state_slot("a"), cm.state_slot("b")], dtype=torch.int32))
    view["right"].state[cm.state_slot("a")] = 1.0
    was = cm.state_slot("a")
    cm.release_passed("a")
    free = cm.free_pages()
    assert max(free) > min(free)                              # windows and chunks gave pages back, the causal layer none
    cm.free_request("a")
    cm.reserve_step([("c", 2)])
    assert cm.state_slot("c") == was and float(view["right"].state[was].abs().max()) == 0.0
    cm.check()


# ---- positions -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("base, dims, s", [(40.0, 6, (8.0, 40, 1.0, 4.0)), (900.0, 16, (2.0, 25, 0.5, 3.0)),
                                           (500000.0, 128, (8.0, 8192, 1.0, 4.0)), (10.0, 2, (1.0, 8, 1.0, 2.0)),
                                           (10000.0, 64, (32.0, 300, 2.0, 2.0))])
def test_frequencies_by_wavelength(base, dims, s):
    scaling = dict(zip(("factor", "original", "low", "high"), s))
    got = RopeWavelength(dims, base, dims and s[0], s[1], s[2], s[3], dims).inv_freq().double()
    want = torch.tensor(plain.wavelength_frequencies(base, dims, scaling), dtype=F)
    assert torch.allclose(got, want, rtol=1e-6)
    plain_f = torch.tensor(plain.frequencies(base, dims), dtype=F)
    assert (want <= plain_f * (1 + 1e-12)).all() and (want >= plain_f / s[0] * (1 - 1e-12)).all()
    if dims == 128:                                           # all three regions are there
        ratio = want / plain_f
        assert (ratio == 1).any() and (ratio < 0.126).any() and ((ratio > 0.13) & (ratio < 0.99)).any()


def test_stretched_frequencies_and_their_multiplier():
    s = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}
    part = RopeStretched(32, 500.0, 4.0, 64, 8.0, 1.0, 16)
    assert torch.allclose(part.inv_freq().double(), torch.tensor(plain.yarn_frequencies(500.0, 16, s), dtype=F), rtol=1e-6)
    assert part.rotation("cpu").scale == pytest.approx(plain.yarn_multiplier(s)) == pytest.approx(0.1 * math.log(4) + 1)


# ---- the plain mechanisms at their edges ---------------------------------------------------------------
def test_plain_norms_and_activation():
    x = torch.tensor([[1.0, 3.0, 5.0, 7.0]], dtype=F)
    one, zero = torch.ones(4, dtype=F), torch.zeros(4, dtype=F)
    assert torch.allclose(plain.layer_norm(x, one, zero, 0.0), (x - 4) / math.sqrt(5.0))
    assert torch.allclose(plain.layer_norm(x, 2 * one, one, 11.0), (x - 4) / 4.0 * 2 + 1)
    assert plain.relu_squared(torch.tensor([-2.0, 0.0, 3.0])).tolist() == [0.0, 0.0, 9.0]
    w = {"left.out": 2 * one, "right.out": one}
    got = plain.side_by_side(w, "", 7 * torch.ones((1, 4), dtype=F), -3 * torch.ones((1, 4), dtype=F), 0.0)
    assert torch.allclose(got, 0.5 * torch.ones((1, 4), dtype=F))       # (2 - 1) / 2


def test_plain_masks_and_query_factor():
    assert [plain.visible(i, window=3) for i in range(6)] == [0, 0, 0, 1, 2, 3]
    assert [plain.visible(i, window=1) for i in range(3)] == [0, 1, 2]
    assert [plain.visible(i, chunk=3) for i in range(7)] == [0, 0, 0, 3, 3, 3, 6]
    f = plain.temperature(range(9), 0.5, 4).tolist()
    assert f[:3] == [1.0] * 3 and f[3:7] == pytest.approx([1 + 0.5 * math.log(2)] * 4) and f[7] == pytest.approx(1 + 0.5 * math.log(3))


def test_plain_turns():
    x = torch.arange(1.0, 7.0, dtype=F).view(1, 1, 6)
    quarter = [math.pi / 2, 0.0]
    assert torch.allclose(plain.turn(x, torch.tensor([1]), quarter, "neighbours"), torch.tensor([-2.0, 1, 3, 4, 5, 6], dtype=F))
    assert torch.allclose(plain.turn(x, torch.tensor([1]), quarter, "halves"), torch.tensor([-3.0, 2, 1, 4, 5, 6], dtype=F))
    assert torch.allclose(plain.turn(x, torch.tensor([1]), quarter, "neighbours", 2.0), torch.tensor([-4.0, 2, 6, 8, 5, 6], dtype=F))


def test_plain_sink_and_choice():
    q = torch.zeros((2, 1, 4), dtype=F)
    v = torch.ones((2, 1, 3), dtype=F)
    out = plain.attend(q, q, v, 1.0, sink=torch.tensor([math.log(3.0)], dtype=F))
    assert torch.allclose(out, torch.tensor([[1 / 4] * 3, [2 / 5] * 3], dtype=F))
    c = torch.tensor([-0.1, -0.9, -0.2, -0.3, -0.25, -0.28], dtype=F)
    # groups of two: sums -1.0, -0.5, -0.53: the best single value lies in the group that loses
    assert plain.choose(c, 2, 3, 1) == [2, 3] and plain.choose(c, 3, 3, 2) == [2, 4, 5] and plain.choose(c, 2, 1, 1) == [0, 2]
    # one expert a group counts by itself
    assert plain.choose(c, 2, 6, 2) == [0, 2]


def test_plain_experts_by_hand():
    eye = torch.eye(2, dtype=F)
    w = {"router": torch.tensor([[0.0, 0.0], [0.0, 0.0], [math.log(3.0), 0.0]], dtype=F), "correction": torch.tensor([0.5, -1.0, 0.0], dtype=F)}
    for e in range(3):
        w.update({f"e{e}.up": eye * (e + 1), f"e{e}.down": eye})
    m = {"router": {"experts": 3, "top": 2, "scale": 2.0}, "expert": {"ff": 2}}
    # scores 1/2, 1/2, 3/4: the choice takes 0 and 2, with weights 2 (1/2) / (5/4) and 2 (3/4) / (5/4)
    got = plain.experts(w, "", torch.tensor([[1.0, -1.0]], dtype=F), m)
    assert torch.allclose(got, torch.tensor([[0.8 * 1 + 1.2 * 9, 0.0]], dtype=F))


def test_plain_is_causal_and_greedy_continues_it():
    for cfg in (SMALL_A, SMALL_B, SMALL_C):
        w = {k: v.to(F) for k, v in random_weights(cfg, 1).items()}
        tokens = random_tokens(cfg["vocab"], 12, seed=2)
        rows = []
        whole = plain.forward(cfg, w, tokens, rows)
        assert len(rows) == len(cfg["layers"]) and rows[0].shape == (12, cfg["width"])
        for n in (1, 2, 7):
            assert torch.allclose(plain.forward(cfg, w, tokens[:n]), whole[:n], atol=1e-9)
        assert plain.greedy(cfg, w, tokens[:4], 2)[0] == int(whole[3].argmax())


def test_every_mechanism_moves_the_logits():
    """A tensor that is changed shows at the last token: nothing of the configuration is idle."""
    w = {k: v.to(F) for k, v in random_weights(SMALL_A, 3).items()}
    tokens = random_tokens(SMALL_A["vocab"], 40, seed=1)
    base = plain.forward(SMALL_A, w, tokens)
    for name in ("l1.mix.sink", "l1.mix.g", "l2.mix.left.q.norm", "l0.mix.left.k.b", "l0.mix.left.v.b", "l0.mix.right.a2.b",
                 "l2.mix.right.lam", "l1.mlp.correction", "l1.mlp.shared.down", "l0.norm1.b", "l0.mix.right.out", "final.norm.b"):
        moved = plain.forward(SMALL_A, {**w, name: w[name] * -0.5 + 0.3}, tokens)
        assert (moved - base)[-1].abs().max() > 1e-3 * base.abs().max(), name
