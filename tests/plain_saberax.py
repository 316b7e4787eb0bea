"""A plain, slow implementation of the Saberax decoder in float64, one function per mechanism,
written from the design's equations.  It runs one whole sequence at a time on the CPU and shares
no code with the engine; the tests compare the engine with it.

Notation: ``x`` is ``[T, width]``, a linear weight is stored ``[out, in]`` and applied as ``x @ W.T``;
``cfg`` is the dictionary of ``config.json`` and ``w`` maps tensor names to float64 tensors.
"""
from __future__ import annotations

import json
import math
import os
import struct

import torch

F = torch.float64


def load_folder(folder: str):
    """Configuration and float64 tensors of a model folder, read with the standard library and torch alone."""
    with open(os.path.join(folder, "config.json")) as fh:
        cfg = json.load(fh)
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}
    with open(os.path.join(folder, "model.safetensors"), "rb") as fh:
        (n,) = struct.unpack("<Q", fh.read(8))
        header = json.loads(fh.read(n))
        data = fh.read()
    weights = {}
    for name, ent in header.items():
        if name != "__metadata__":
            lo, hi = ent["data_offsets"]
            weights[name] = torch.frombuffer(bytearray(data[lo:hi]), dtype=kinds[ent["dtype"]]).view(ent["shape"]).to(F)
    return cfg, weights


# ---- small pieces ---------------------------------------------------------------------------------
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


def time_conv(u, taps_w, bias):
    """``y_t = bias + sum_j w[:, j] u_(t - taps + 1 + j)`` with zeros before the start; ``taps_w`` is ``[channels, taps]``."""
    t, taps = u.shape[0], taps_w.shape[1]
    y = bias.expand(u.shape).clone()
    for i in range(t):
        for j in range(taps):
            src = i - taps + 1 + j
            if src >= 0:
                y[i] += taps_w[:, j] * u[src]
    return y


def block_diagonal(u, mats, bias):
    """``blocks`` square matrices ``[out, in]`` on equal consecutive parts of ``u``, a bias per output."""
    n = mats.shape[1]
    return torch.cat([u[:, b * n:(b + 1) * n] @ mats[b].T + bias[b] for b in range(mats.shape[0])], dim=1)


# ---- positions ------------------------------------------------------------------------------------
def frequencies(base, dims):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_frequencies(base, dims, s):
    """Frequencies that turn fast stay, slow ones are divided by ``factor``, a ramp over the pair's index between."""
    def at(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(frequencies(base, dims)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out


def yarn_multiplier(s):
    return 0.1 * math.log(s["factor"]) + 1.0


def wavelength_frequencies(base, dims, s):
    """Frequencies of short wavelengths stay, those of long ones are divided by ``factor``, a blend between."""
    out = []
    for f in frequencies(base, dims):
        wave = 2.0 * math.pi / f
        if wave < s["original"] / s["high"]:
            out.append(f)
        elif wave > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            mix = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1.0 - mix) * f / s["factor"] + mix * f)
    return out


def turn(x, pos, freq, pairs, mult=1.0):
    """``x [T, heads, dim]``: the first ``2 len(freq)`` elements of every head turned pair by pair; ``pairs`` is
    ``"neighbours"`` (2i with 2i + 1) or ``"halves"`` (i with i + n/2).  Cosine and sine carry ``mult``."""
    out = x.clone()
    n = len(freq)
    for i in range(n):
        a, b = (2 * i, 2 * i + 1) if pairs == "neighbours" else (i, i + n)
        ang = pos.to(F) * freq[i]
        c, s = (torch.cos(ang) * mult).view(-1, 1), (torch.sin(ang) * mult).view(-1, 1)
        out[:, :, a] = x[:, :, a] * c - x[:, :, b] * s
        out[:, :, b] = x[:, :, b] * c + x[:, :, a] * s
    return out


def temperature(pos, coef, every):
    """A factor on the query at every position."""
    return torch.tensor([1.0 + coef * math.log(math.floor((int(p) + 1) / every) + 1) for p in pos], dtype=F)


# ---- attention ------------------------------------------------------------------------------------
def visible(i, window=None, chunk=None):
    """First key that position ``i`` sees; the last one is ``i`` itself."""
    lo = 0
    if window is not None:
        lo = max(lo, i - window + 1)
    if chunk is not None:
        lo = max(lo, (i // chunk) * chunk)
    return lo


def attend(q, k, v, scale, window=None, chunk=None, sink=None):
    """Softmax attention of every position over the keys it sees; ``sink`` (per head) is one more term of the
    denominator, ``exp(sink)``, without a key or a value."""
    t, nh, ng = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros((t, nh, v.shape[2]), dtype=F)
    for a in range(nh):
        g = a // (nh // ng)
        for i in range(t):
            lo = visible(i, window, chunk)
            s = (k[lo:i + 1, g] @ q[i, a]) * scale
            if sink is not None:
                p = torch.softmax(torch.cat([s, sink[a].view(1)]), dim=0)[:-1]
            else:
                p = torch.softmax(s, dim=0)
            out[i, a] = p @ v[lo:i + 1, g]
    return out.reshape(t, -1)


def temperature_attention(w, p, h, m, eps):
    """Causal attention without a turn: heads normed with a weight, queries times a factor of their position."""
    t, nh, ng, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = unit_rms((h @ w[p + "q"].T).view(t, nh, d), eps) * w[p + "q.norm"]
    k = unit_rms((h @ w[p + "k"].T).view(t, ng, d), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(t, ng, m["vdim"])
    q = q * temperature(range(t), m["q_temp"]["coef"], m["q_temp"]["every"]).view(-1, 1, 1)
    return attend(q, k, v, m["scale"]) @ w[p + "o"].T


def window_attention(w, p, h, m, eps):
    """Attention in a sliding window: biases, neighbouring pairs turned by stretched frequencies, then unit heads."""
    t, nh, ng, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(t)
    freq = yarn_frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"]["scaling"])
    mult = yarn_multiplier(m["rot"]["scaling"])
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(t, nh, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(t, ng, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(t, ng, m["vdim"])
    q = unit_rms(turn(q, pos, freq, "neighbours", mult), eps)
    k = unit_rms(turn(k, pos, freq, "neighbours", mult), eps)
    return attend(q, k, v, m["scale"], window=m["mask"]["size"]) @ w[p + "o"].T


def chunk_attention(w, p, h, m, eps):
    """Attention inside chunks of positions with a sink: values are the projected keys, halves turned by scaled
    frequencies, then unit heads, and a gate per head."""
    t, nh, ng, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(t)
    freq = wavelength_frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"]["scaling"])
    q, k = (h @ w[p + "q"].T).view(t, nh, d), (h @ w[p + "k"].T).view(t, ng, d)
    v = k
    q, k = unit_rms(turn(q, pos, freq, "halves"), eps), unit_rms(turn(k, pos, freq, "halves"), eps)
    out = attend(q, k, v, m["scale"], chunk=m["mask"]["size"], sink=w[p + "sink"]).view(t, nh, d)
    gate = torch.sigmoid(h @ w[p + "g"].T)
    return (out * gate.unsqueeze(-1)).reshape(t, nh * d) @ w[p + "o"].T


# ---- recurrences ----------------------------------------------------------------------------------
def rglru(w, p, h, m):
    """Two branches: a gelu of one product, and a time convolution of another that passes a linear recurrence
    per channel whose decay and input gate come from block-diagonal products."""
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = time_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = torch.sigmoid(block_diagonal(u, w[p + "ra"], w[p + "ra.b"]))
    i = torch.sigmoid(block_diagonal(u, w[p + "ri"], w[p + "ri.b"]))
    lam = w[p + "lam"]
    log_a = -8.0 * r * (torch.log1p(torch.exp(-lam.abs())) + torch.clamp(lam, min=0.0))
    s, rows = torch.zeros_like(u[0]), []
    for t in range(h.shape[0]):
        s = torch.exp(log_a[t]) * s + torch.sqrt(-torch.expm1(2.0 * log_a[t])) * i[t] * u[t]
        rows.append(s)
    return (torch.stack(rows) * y) @ w[p + "o"].T


def gla(w, p, h, m, eps):
    """Gated linear attention: a matrix state per head whose key rows decay each by a factor of their own."""
    t, nh, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(t, nh, d) * d ** -0.5
    k, v = (h @ w[p + "k"].T).view(t, nh, d), (h @ w[p + "v"].T).view(t, nh, dv)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    alpha = (torch.sigmoid(z) ** (1.0 / m["tau"])).view(t, nh, d)
    out = torch.zeros((t, nh, dv), dtype=F)
    for a in range(nh):
        s = torch.zeros((d, dv), dtype=F)
        for i in range(t):
            s = alpha[i, a].view(-1, 1) * s + torch.outer(k[i, a], v[i, a])
            out[i, a] = s.T @ q[i, a]
    out = unit_rms(out, eps) * w[p + "norm"]
    return (out.reshape(t, nh * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- the layer's parts ------------------------------------------------------------------------------
def side_by_side(w, p, left, right, eps):
    """Half the sum of two mixers' outputs, each normed over the width with a weight."""
    return 0.5 * (unit_rms(left, eps) * w[p + "left.out"] + unit_rms(right, eps) * w[p + "right.out"])


def mixer(cfg, w, entry, p, h):
    m, eps = entry["mixer"], cfg["norm"]["eps"]
    if entry["type"] == "attention":
        return chunk_attention(w, p, h, m, eps)
    if entry["type"] == "parallel":
        return side_by_side(w, p, temperature_attention(w, p + "left.", h, m["left"], eps),
                            rglru(w, p + "right.", h, m["right"]), eps)
    return side_by_side(w, p, window_attention(w, p + "left.", h, m["left"], eps),
                        gla(w, p + "right.", h, m["right"], eps), eps)


def choose(choice, top, count, keep):
    """The ``top`` outputs of one row by their choice scores inside the ``keep`` groups whose two largest sum highest
    (ties: the lower index)."""
    n = choice.shape[0] // count
    value = [sum(sorted(choice[g * n:(g + 1) * n].tolist(), reverse=True)[:2]) for g in range(count)]
    kept = sorted(range(count), key=lambda g: (-value[g], g))[:keep]
    open_ = [e for g in kept for e in range(g * n, (g + 1) * n)]
    return sorted(open_, key=lambda e: (-float(choice[e]), e))[:top]


def experts(w, p, h, m):
    """A sigmoid router with a correction of the choice, groups, weights brought to a sum; a shared expert beside."""
    r = m["router"]
    scores = torch.sigmoid(h @ w[p + "router"].T)
    groups = r.get("groups") or {"count": 1, "keep": 1}
    expert = lambda q, x: relu_squared(x @ w[q + "up"].T) @ w[q + "down"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids = choose(scores[t] + w[p + "correction"], r["top"], groups["count"], groups["keep"])
        total = sum(float(scores[t, e]) for e in ids) + 1e-20
        for e in ids:
            out[t] += float(scores[t, e]) / total * r["scale"] * expert(f"{p}e{e}.", h[t])
    if m.get("shared") is not None:
        out = out + expert(p + "shared.", h)
    return out


def feed_forward(w, p, h, m):
    if m["kind"] == "dense":
        return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T
    return experts(w, p, h, m)


def tensors_of(cfg, i):
    """The layer whose tensors layer ``i`` uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def layer(cfg, w, i, x):
    entry, p, eps, m = cfg["layers"][i], f"l{tensors_of(cfg, i)}.", cfg["norm"]["eps"], cfg["residual_mult"]
    x = x + m * mixer(cfg, w, entry, p + "mix.", layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps))
    if entry.get("mlp") is not None:
        x = x + m * feed_forward(w, p + "mlp.", layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps), entry["mlp"])
    return x


def forward(cfg, w, tokens, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` (a list) receives the rows behind every layer."""
    x = w["embed"][torch.as_tensor(list(tokens), dtype=torch.long)]
    for i in range(len(cfg["layers"])):
        x = layer(cfg, w, i, x)
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"]) @ w["head"].T


def greedy(cfg, w, prompt, n):
    """``n`` tokens by argmax, each from a whole pass over everything so far."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(torch.argmax(forward(cfg, w, tokens)[-1])))
    return tokens[len(prompt):]
