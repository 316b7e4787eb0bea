"""Small Vametar configurations with random weights, written as model folders by the tests.

The weights are drawn here with torch's generator (not with the package's), large enough that every
mechanism moves the logits: decays between fast and slow, gates on both sides of their middle, shifts
and value shares of either sign, a bigram table as large as the embedding.  Everything is stored in
bfloat16, so the plain implementation and the engine read the same values.
"""
from __future__ import annotations

import json
import os

import torch

from tinyinfer_b200.weights.safetensors_io import write_safetensors


def attention(heads, kv_heads, dim, vdim, rot_dims, base, scale, v_mix=False):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "rot": {"dims": rot_dims, "base": base}, "v_mix": v_mix}}


def rglru(width, blocks, conv):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def gla(heads, dim, vdim, tau):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def layer(entry, ff=None):
    return dict(entry, mlp=None if ff is None else {"kind": "dense", "ff": ff})


def model(vocab, width, bigram, eps, mult, scale, layers):
    buckets, prev, cur = bigram
    return {"architecture": "Vametar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": prev, "mul_cur": cur}}, "logit_scale": scale,
            "layers": layers}


# every size differs between the parts: fewer kv heads than heads, value heads of another size, turns over
# part of a head, values mixed over three layers with a layer that does not mix between them, feed-forwards
# behind every kind of mixer and behind none
SMALL_A = model(131, 48, (37, 1009, 11), 1e-6, 0.8, 1.7, [
    layer(rglru(60, 3, 3), 40),
    layer(attention(4, 2, 12, 8, 6, 1000.0, 0.29, v_mix=True)),
    layer(gla(3, 8, 20, 9.0), 32),
    layer(attention(2, 1, 16, 24, 16, 50.0, 0.2), 24),
    layer(attention(6, 1, 10, 16, 4, 300.0, 0.31, v_mix=True), 56),
    layer(rglru(20, 5, 2)),
    layer(attention(4, 4, 8, 4, 8, 20.0, 0.35, v_mix=True))])
# values that make branches coincide or vanish: one bucket, factors 0 and 1, one head, one block, one tap,
# a block per channel, no turn, a layer that mixes values alone, the factors 1
SMALL_B = model(97, 36, (1, 0, 1), 1e-5, 1.0, 1.0, [
    layer(attention(1, 1, 16, 16, 0, 1.0, 0.25, v_mix=True), 36),
    layer(rglru(36, 1, 1)),
    layer(gla(1, 16, 16, 1.0), 8),
    layer(rglru(8, 8, 6), 16),
    layer(attention(3, 3, 8, 8, 2, 30.0, 0.35))])
# sizes that tensor-core kernels take, value heads wider than a block of state columns
SMALL_C = model(1009, 128, (211, 13, 5), 2e-6, -0.6, 0.9, [
    layer(attention(4, 2, 64, 64, 32, 20000.0, 0.125, v_mix=True), 192),
    layer(rglru(192, 3, 4), 128),
    layer(gla(2, 64, 192, 16.0)),
    layer(attention(2, 1, 128, 128, 128, 300000.0, 0.09, v_mix=True), 256),
    layer(gla(4, 128, 32, 5.0), 64),
    layer(rglru(128, 8, 2))])
# no attention at all: nothing is paged
SMALL_D = model(64, 32, (16, 3, 2), 1e-5, 0.5, 3.0, [layer(gla(2, 12, 8, 4.0), 24), layer(rglru(24, 2, 4))])
SMALL = {"A": SMALL_A, "B": SMALL_B, "C": SMALL_C, "D": SMALL_D}


def mixer_weights(kind: str, m: dict, width: int, g: torch.Generator, v_mix: bool = True) -> dict:
    """Tensors of one mixer under their local names."""
    def mat(rows, cols, gain=1.0):
        return (torch.randn((rows, cols), generator=g) * gain / cols ** 0.5).to(torch.bfloat16)

    def vec(n, std, mean=0.0):
        return (mean + torch.randn((n,), generator=g) * std).to(torch.bfloat16)

    if kind == "attention":
        nq, nk, nv = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
        w = {"q": mat(nq, width, 2.0), "k": mat(nk, width, 2.0), "v": mat(nv, width), "q.norm": vec(nq, 0.3, 1.5),
             "k.norm": vec(nk, 0.3, 1.5), "o": mat(width, m["heads"] * m["vdim"])}
        if v_mix:
            w["vmix"] = torch.tensor(float(torch.rand((), generator=g)) * 1.4 - 0.2).to(torch.bfloat16)
        return w
    if kind == "rglru":
        n, blocks, taps = m["width"], m["blocks"], m["conv"]
        per = n // blocks
        conv = torch.randn((n, taps), generator=g) * 0.6 + (torch.arange(taps) == taps - 1) * 0.8
        square = lambda: (torch.randn((blocks, per, per), generator=g) * 2.0 / per ** 0.5).to(torch.bfloat16)
        return {"y": mat(n, width, 1.5), "y.b": vec(n, 0.5), "x": mat(n, width, 1.5), "x.b": vec(n, 0.5),
                "conv": conv.to(torch.bfloat16), "conv.b": vec(n, 0.3), "ra": square(), "ra.b": vec(n, 0.5).view(blocks, per),
                "ri": square(), "ri.b": vec(n, 0.5).view(blocks, per), "lam": vec(n, 2.0, -3.5), "o": mat(width, n, 1.5)}
    nk, nv, rank = m["heads"] * m["dim"], m["heads"] * m["vdim"], max(1, width // 5)
    return {"q": mat(nk, width, 2.0), "k": mat(nk, width), "v": mat(nv, width), "g": mat(nv, width, 2.0),
            "a1": mat(rank, width), "a2": mat(nk, rank, 2.0), "a2.b": vec(nk, 1.5, 1.0), "norm": vec(m["vdim"], 0.2, 1.0),
            "o": mat(width, nv)}


def mlp_weights(ff: int, width: int, g: torch.Generator) -> dict:
    mat = lambda rows, cols, gain: (torch.randn((rows, cols), generator=g) * gain / cols ** 0.5).to(torch.bfloat16)
    return {"gate": mat(ff, width, 2.0), "up": mat(ff, width, 2.0), "down": mat(width, ff, 1.0)}


def random_weights(cfg: dict, seed: int) -> dict:
    g = torch.Generator().manual_seed(seed)
    width, vocab = cfg["width"], cfg["vocab"]
    norm = lambda: torch.tensor(0.8 + 0.6 * float(torch.rand((), generator=g))).to(torch.bfloat16)
    table = lambda rows: (torch.randn((rows, width), generator=g) * 0.5).to(torch.bfloat16)
    gate = lambda: (torch.randn((width, width), generator=g) * 2.0 / width ** 0.5).to(torch.bfloat16)
    vec = lambda std: (torch.randn((width,), generator=g) * std).to(torch.bfloat16)
    w = {"embed": table(vocab), "bigram": table(cfg["embedding"]["bigram"]["buckets"] + 1), "head": table(vocab),
         "final.norm": norm()}
    for i, entry in enumerate(cfg["layers"]):
        p = f"l{i}."
        w.update({p + "norm1": norm(), p + "shift": vec(0.5), p + "rg1": gate(), p + "rg1.b": vec(0.7)})
        for name, t in mixer_weights(entry["type"], entry["mixer"], width, g, entry["mixer"].get("v_mix", False)).items():
            w[p + "mix." + name] = t
        if entry["mlp"] is not None:
            w.update({p + "norm2": norm(), p + "rg2": gate(), p + "rg2.b": vec(0.7)})
            for name, t in mlp_weights(entry["mlp"]["ff"], width, g).items():
                w[p + "mlp." + name] = t
    return w


def write_model(folder: str, cfg: dict, seed: int) -> str:
    os.makedirs(folder, exist_ok=True)
    write_safetensors(os.path.join(folder, "model.safetensors"), random_weights(cfg, seed))
    with open(os.path.join(folder, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    return folder


def make_model(tmp_path, name: str, seed: int = 11) -> str:
    d = os.path.join(str(tmp_path), f"vametar_{name}_{seed}")
    if not os.path.isdir(d):
        write_model(d, SMALL[name], seed)
    return d


def drawn_configuration(seed: int) -> dict:
    """A configuration whose every size, constant, option and order of layers is drawn from ``seed``."""
    import random
    r = random.Random(seed)
    pick = r.choice
    width = pick([16, 24, 40, 64, 72])
    values = pick([6, 8, 24, 32])                 # elements of the values that layers mix: one number for all of them
    layers = []
    for _ in range(r.randint(1, 6)):
        kind = pick(["attention", "rglru", "gla"])
        if kind == "attention":
            kv = pick([1, 2])
            dim, v_mix = pick([4, 6, 10, 16, 32, 48]), r.random() < 0.6
            vdim = values // kv if v_mix else pick([2, 5, 8, 16, 40])
            entry = attention(kv * pick([1, 2, 3]), kv, dim, vdim, pick([0, 2, dim // 2 // 2 * 2, dim]),
                              pick([10.0, 500.0, 250000.0]), r.uniform(0.05, 0.4), v_mix=v_mix)
        elif kind == "rglru":
            blocks = pick([1, 2, 3, 4])
            entry = rglru(blocks * pick([1, 3, 8, 16, 20]), blocks, pick([1, 2, 3, 4, 7]))
        else:
            entry = gla(pick([1, 2, 3, 5]), pick([3, 8, 16, 36]), pick([5, 8, 16, 24]), pick([1.0, 3.5, 16.0]))
        layers.append(layer(entry, None if r.random() < 0.35 else pick([8, 24, 31, 48])))
    buckets = pick([1, 2, 29, 500])
    return model(pick([33, 100, 257]), width, (buckets, r.randint(0, 5000), r.randint(0, 5000)), pick([1e-6, 1e-5]),
                 r.uniform(0.3, 1.2), r.uniform(0.5, 3.0), layers)


def make_drawn_model(tmp_path, seed: int) -> str:
    d = os.path.join(str(tmp_path), f"vametar_drawn_{seed}")
    return d if os.path.isdir(d) else write_model(d, drawn_configuration(seed), seed)
