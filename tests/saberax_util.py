"""Small Saberax configurations with random weights, written as model folders by the tests.

The weights are drawn here with torch's generator (not with the package's), large enough that every
mechanism moves the logits: biases as large as the projections, sinks on both sides of the scores, decays
between fast and slow, corrections that change the experts' order.  Everything is stored in bfloat16, so
the plain implementation and the engine read the same values.
"""
from __future__ import annotations

import json
import os

import torch

from tinyinfer_b200.weights.safetensors_io import write_safetensors


# ---- configurations -----------------------------------------------------------------------------
def attention(heads, kv_heads, dim, chunk, rot, scale, base, scaling):
    """``scaling``: (factor, original, low, high)."""
    s = dict(zip(("factor", "original", "low", "high"), scaling))
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                                           "mask": {"size": chunk}, "rot": {"dims": rot, "base": base, "scaling": s}}}


def rising(heads, kv_heads, dim, vdim, scale, coef, every, width, blocks, conv):
    """Causal attention with a rising query factor beside a recurrence per channel."""
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                 "q_temp": {"coef": coef, "every": every}},
        "right": {"width": width, "blocks": blocks, "conv": conv}}}


def windowed(heads, kv_heads, dim, vdim, window, rot, scale, base, scaling, gla):
    """Attention in a window beside gated linear attention; ``scaling``: (factor, original, fast, slow), ``gla``:
    (heads, dim, vdim, tau)."""
    s = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "parallel_2", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window},
                 "rot": {"dims": rot, "base": base, "scaling": s}},
        "right": dict(zip(("heads", "dim", "vdim", "tau"), gla))}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale, groups=None, shared=None):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def layer(entry, mlp=None, weights_of=None):
    out = dict(entry, mlp=mlp)
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


def model(vocab, width, eps, mult, layers):
    return {"architecture": "Saberax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": layers}


# every size differs between the parts: fewer kv heads than heads, value heads of another size, turns over part of a
# head, windows and chunks that are no multiples of a page, every kind of feed-forward behind some mixer and none
# behind another, a layer whose tensors run a second time in front of and behind other layers
SMALL_A = model(131, 48, 1e-6, 0.6, [
    layer(windowed(4, 2, 12, 8, 21, 8, 0.5, 500.0, (4.0, 32, 8.0, 1.0), (3, 8, 20, 9.0)), dense(40)),
    layer(attention(4, 2, 10, 19, 6, 0.6, 40.0, (8.0, 40, 1.0, 4.0)), moe(12, 3, 24, 1.7, groups=(3, 2), shared=40)),
    layer(rising(6, 3, 8, 12, 0.3, 0.4, 9, 60, 3, 3), moe(8, 2, 16, 2.5, groups=(2, 1))),
    layer(attention(3, 1, 16, 33, 16, 0.4, 900.0, (2.0, 25, 0.5, 3.0))),
    layer(rising(6, 3, 8, 12, 0.3, 0.4, 9, 60, 3, 3), moe(8, 2, 16, 2.5, groups=(2, 1)), weights_of=2),
    layer(windowed(2, 2, 16, 24, 5, 16, 0.4, 90.0, (2.0, 64, 4.0, 0.5), (2, 12, 6, 3.0)), dense(56))])
# values that make branches coincide or vanish: one head, one block, one tap, a window of the token itself, chunks of
# one token, the factors 1, no turn, one group, no shared expert, all experts chosen, a constant query
SMALL_B = model(97, 36, 1e-5, 1.0, [
    layer(windowed(1, 1, 16, 16, 1, 0, 0.25, 2.0, (1.0, 1, 1.0, 1.0), (1, 16, 16, 1.0)), moe(4, 4, 12, 1.0)),
    layer(attention(2, 2, 8, 1, 2, 1.0, 7.0, (1.0, 8, 1.0, 2.0)), dense(36)),
    layer(rising(1, 1, 6, 5, 0.4, 0.0, 1, 20, 1, 1)),
    layer(rising(3, 3, 7, 7, 0.4, 1.5, 1, 12, 12, 6), moe(5, 1, 9, 3.0, groups=(1, 1), shared=7)),
    layer(windowed(2, 1, 9, 4, 64, 4, 0.3, 10.0, (3.0, 16, 2.0, 1.0), (1, 5, 9, 2.5)), dense(8))])
# sizes that tensor-core kernels take
SMALL_C = model(1009, 128, 2e-6, -0.8, [
    layer(windowed(4, 2, 64, 64, 50, 32, 0.125, 20000.0, (4.0, 128, 16.0, 1.0), (2, 64, 128, 16.0)), dense(192)),
    layer(rising(4, 2, 48, 32, 0.15, 0.2, 40, 192, 3, 4), moe(16, 4, 64, 2.0, groups=(4, 2), shared=128)),
    layer(attention(4, 4, 64, 80, 64, 0.2, 300000.0, (8.0, 64, 1.0, 4.0)), moe(8, 2, 96, 1.5, groups=(2, 1), shared=64)),
    layer(windowed(2, 1, 128, 32, 130, 128, 0.09, 5000.0, (2.0, 256, 32.0, 1.0), (4, 32, 32, 4.0)), dense(256)),
    layer(attention(4, 4, 64, 80, 64, 0.2, 300000.0, (8.0, 64, 1.0, 4.0)), moe(8, 2, 96, 1.5, groups=(2, 1), shared=64),
          weights_of=2)])
SMALL = {"A": SMALL_A, "B": SMALL_B, "C": SMALL_C}


# ---- weights ------------------------------------------------------------------------------------
def _mat(g, rows, cols, gain=1.0):
    return (torch.randn((rows, cols), generator=g) * gain / cols ** 0.5).to(torch.bfloat16)


def _vec(g, n, std, mean=0.0):
    return (mean + torch.randn((n,), generator=g) * std).to(torch.bfloat16)


def heads_weights(m: dict, width: int, g: torch.Generator, values: bool = True) -> dict:
    nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
    w = {"q": _mat(g, nq, width, 2.0), "k": _mat(g, nk, width, 2.0), "o": _mat(g, width, m["heads"] * m["vdim"])}
    if values:
        w["v"] = _mat(g, m["kv_heads"] * m["vdim"], width, 1.5)
    return w


def mixer_weights(kind: str, m: dict, width: int, g: torch.Generator) -> dict:
    """Tensors of one mixer under their local names."""
    if kind == "attention":
        return {**heads_weights(m, width, g, values=False), "sink": _vec(g, m["heads"], 1.5),
                "g": _mat(g, m["heads"], width, 2.0)}
    a, b = m["left"], m["right"]
    w = {"left." + n: t for n, t in heads_weights(a, width, g).items()}
    w.update({"left.out": _vec(g, width, 0.3, 1.0), "right.out": _vec(g, width, 0.3, 1.0)})
    if kind == "parallel":
        w.update({"left.q.norm": _vec(g, a["dim"], 0.3, 1.0), "left.k.norm": _vec(g, a["dim"], 0.3, 1.2)})
        n, blocks, taps = b["width"], b["blocks"], b["conv"]
        per = n // blocks
        conv = torch.randn((n, taps), generator=g) * 0.6 + (torch.arange(taps) == taps - 1) * 0.8
        square = lambda: (torch.randn((blocks, per, per), generator=g) * 2.0 / per ** 0.5).to(torch.bfloat16)
        right = {"y": _mat(g, n, width, 1.5), "y.b": _vec(g, n, 0.5), "x": _mat(g, n, width, 1.5), "x.b": _vec(g, n, 0.5),
                 "conv": conv.to(torch.bfloat16), "conv.b": _vec(g, n, 0.3), "ra": square(),
                 "ra.b": _vec(g, n, 0.5).view(blocks, per), "ri": square(), "ri.b": _vec(g, n, 0.5).view(blocks, per),
                 "lam": _vec(g, n, 2.0, -3.5), "o": _mat(g, width, n, 1.5)}
    else:
        for name in ("q", "k", "v"):
            w[f"left.{name}.b"] = _vec(g, w["left." + name].shape[0], 1.0)
        nk, nv, rank = b["heads"] * b["dim"], b["heads"] * b["vdim"], max(1, width // 5)
        right = {"q": _mat(g, nk, width, 2.0), "k": _mat(g, nk, width), "v": _mat(g, nv, width), "g": _mat(g, nv, width, 2.0),
                 "a1": _mat(g, rank, width), "a2": _mat(g, nk, rank, 2.0), "a2.b": _vec(g, nk, 1.5, 1.0),
                 "norm": _vec(g, b["vdim"], 0.2, 1.0), "o": _mat(g, width, nv)}
    w.update({"right." + n: t for n, t in right.items()})
    return w


def mlp_weights(mlp: dict, width: int, g: torch.Generator) -> dict:
    if mlp["kind"] == "dense":
        return {"gate": _mat(g, mlp["ff"], width, 2.0), "up": _mat(g, mlp["ff"], width, 2.0), "down": _mat(g, width, mlp["ff"])}
    r, ff = mlp["router"], mlp["expert"]["ff"]
    # corrections larger than the scores' spread, of either sign: the choice is not the plain order of the scores,
    # choice scores fall below zero, and few choices are so close that rounding turns them
    w = {"router": _mat(g, r["experts"], width, 2.0), "correction": _vec(g, r["experts"], 1.0, -0.3)}
    for e in range(r["experts"]):
        w.update({f"e{e}.up": _mat(g, ff, width, 1.0), f"e{e}.down": _mat(g, width, ff, 0.7)})
    if mlp.get("shared") is not None:
        w.update({"shared.up": _mat(g, mlp["shared"]["ff"], width, 1.2), "shared.down": _mat(g, width, mlp["shared"]["ff"])})
    return w


def norm_weights(name: str, width: int, g: torch.Generator) -> dict:
    return {name: _vec(g, width, 0.2, 1.0), name + ".b": _vec(g, width, 0.3)}


def random_weights(cfg: dict, seed: int) -> dict:
    g = torch.Generator().manual_seed(seed)
    width = cfg["width"]
    # a mean and a scale of their own per row, so that a norm without either would show
    rows = torch.randn((cfg["vocab"], width), generator=g) * (0.3 + torch.rand((cfg["vocab"], 1), generator=g))
    w = {"embed": (rows + torch.randn((cfg["vocab"], 1), generator=g) * 0.5).to(torch.bfloat16),
         "head": _mat(g, cfg["vocab"], width, 3.0), **norm_weights("final.norm", width, g)}
    for i, entry in enumerate(cfg["layers"]):
        if entry.get("weights_of") is not None:
            continue
        p = f"l{i}."
        w.update(norm_weights(p + "norm1", width, g))
        for name, t in mixer_weights(entry["type"], entry["mixer"], width, g).items():
            w[p + "mix." + name] = t
        if entry["mlp"] is not None:
            w.update(norm_weights(p + "norm2", width, g))
            for name, t in mlp_weights(entry["mlp"], width, g).items():
                w[p + "mlp." + name] = t
    return w


def write_model(folder: str, cfg: dict, seed: int) -> str:
    os.makedirs(folder, exist_ok=True)
    write_safetensors(os.path.join(folder, "model.safetensors"), random_weights(cfg, seed))
    with open(os.path.join(folder, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    return folder


def make_model(tmp_path, name: str, seed: int = 11) -> str:
    d = os.path.join(str(tmp_path), f"saberax_{name}_{seed}")
    return d if os.path.isdir(d) else write_model(d, SMALL[name], seed)


def drawn_configuration(seed: int) -> dict:
    """A configuration whose every size, constant and order of layers is drawn from ``seed``."""
    import random
    r = random.Random(seed)
    pick = r.choice
    width = pick([16, 24, 40, 64, 72])

    def heads():
        kv = pick([1, 2, 3])
        return kv * pick([1, 2, 3]), kv, pick([4, 6, 10, 16, 32, 48])

    def drawn_mlp():
        kind = r.random()
        if kind < 0.25:
            return None
        if kind < 0.5:
            return dense(pick([8, 24, 31, 48]))
        count, per = pick([1, 2, 3, 4]), pick([2, 3, 5])
        keep = r.randint(1, count)
        return moe(count * per, r.randint(1, min(per * keep, 4)), pick([8, 15, 32]), pick([0.5, 1.0, 3.0]), groups=(count, keep),
                   shared=pick([None, 8, 40]))

    layers = []
    for i in range(r.randint(1, 6)):
        kind = pick(["attention", "parallel", "parallel_2", "again"])
        own = [j for j, la in enumerate(layers) if "weights_of" not in la]
        if kind == "again" and own:
            j = pick(own)
            layers.append(dict(layers[j], weights_of=j))
            continue
        h, kv, dim = heads()
        rot = pick([0, 2, dim // 2 // 2 * 2, dim])
        if kind == "attention":
            entry = attention(h, kv, dim, pick([1, 2, 7, 16, 33, 64, 200]), rot, r.uniform(0.1, 0.6), pick([10.0, 500.0, 250000.0]),
                              (pick([1.0, 2.0, 8.0]), pick([8, 64, 512]), pick([0.5, 1.0]), pick([2.0, 4.0])))
        elif kind == "parallel":
            blocks = pick([1, 2, 3, 4])
            entry = rising(h, kv, dim, pick([2, 5, 8, 16, 40]), r.uniform(0.05, 0.4), r.uniform(0.0, 1.0), pick([1, 3, 16, 50]),
                           blocks * pick([1, 3, 8, 16, 20]), blocks, pick([1, 2, 3, 4, 7]))
        else:
            entry = windowed(h, kv, dim, pick([2, 5, 8, 16, 40]), pick([1, 2, 5, 16, 17, 33, 64, 200]), rot, r.uniform(0.1, 0.6),
                             pick([10.0, 500.0, 250000.0]), (pick([1.0, 2.0, 8.0]), pick([8, 64, 512]), pick([32.0, 4.0]), pick([1.0, 2.0])),
                             (pick([1, 2, 3, 5]), pick([3, 8, 16, 36]), pick([5, 8, 16, 24]), pick([1.0, 3.5, 16.0])))
        layers.append(layer(entry, drawn_mlp()))
    return model(pick([33, 100, 257]), width, pick([1e-6, 1e-5]), r.uniform(0.3, 1.2), layers)


def make_drawn_model(tmp_path, seed: int) -> str:
    d = os.path.join(str(tmp_path), f"saberax_drawn_{seed}")
    return d if os.path.isdir(d) else write_model(d, drawn_configuration(seed), seed)
