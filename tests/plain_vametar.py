"""A plain, slow implementation of the Vametar decoder in float64, one function per mechanism,
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


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def bigram_rows(tokens, mul_prev, mul_cur, buckets):
    """The bigram table's row of every token: a hash of (token before, token), the last row for the first token."""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + tokens[i] * mul_cur) % buckets for i in range(len(tokens))]


def embed(cfg, w, tokens):
    b = cfg["embedding"]["bigram"]
    rows = bigram_rows([int(t) for t in tokens], b["mul_prev"], b["mul_cur"], b["buckets"])
    return w["embed"][torch.as_tensor(tokens, dtype=torch.long)] + w["bigram"][torch.as_tensor(rows, dtype=torch.long)]


def token_shift(h, mu):
    """``h_t + (h_(t-1) - h_t) mu``, with zeros in front of the first row."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], dim=0)
    return h + (before - h) * mu


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


def frequencies(base, dims):
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)


def turn_halves(x, pos, freq):
    """Turn elements i and i + n/2 of the first n = 2 len(freq) elements of every head of ``x [T, heads, dim]``."""
    out = x.clone()
    half = freq.shape[0]
    ang = (pos.to(F).reshape(-1, 1) * freq.reshape(1, -1)).reshape(x.shape[0], 1, half)
    c, s = torch.cos(ang), torch.sin(ang)
    a, b = x[..., :half], x[..., half:2 * half]
    out[..., :half] = a * c - b * s
    out[..., half:2 * half] = b * c + a * s
    return out


def block_diagonal(u, mats, bias):
    """``blocks`` square matrices ``[out, in]`` on equal consecutive parts of ``u``, a bias per output."""
    n = mats.shape[1]
    return torch.cat([u[:, b * n:(b + 1) * n] @ mats[b].T + bias[b] for b in range(mats.shape[0])], dim=1)


# ---- mixers ---------------------------------------------------------------------------------------
def attention(w, p, h, m, eps, v_first=None):
    """Causal grouped-query attention; the whole query row and the whole key row normed, partly turned heads,
    values mixed with ``v_first`` (the values of an earlier layer) where one is given.  Returns the output
    and the layer's own values before any mixing."""
    t = h.shape[0]
    nh, ng, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]
    k = unit_rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]
    own = h @ w[p + "v"].T
    v = own if v_first is None else (1.0 - w[p + "vmix"]) * own + w[p + "vmix"] * v_first
    q, k, v = q.reshape(t, nh, d), k.reshape(t, ng, d), v.reshape(t, ng, dv)
    pos = torch.arange(t)
    freq = frequencies(float(m["rot"]["base"]), int(m["rot"]["dims"]))
    q, k = turn_halves(q, pos, freq), turn_halves(k, pos, freq)
    out = torch.zeros((t, nh, dv), dtype=F)
    for a in range(nh):
        g = a // (nh // ng)
        for i in range(t):
            out[i, a] = torch.softmax((k[:i + 1, g] @ q[i, a]) * m["scale"], dim=0) @ v[:i + 1, g]
    return out.reshape(t, nh * dv) @ w[p + "o"].T, own


def rglru(w, p, h, m):
    """Two branches: a gelu of one product, and a time convolution of another that passes a linear recurrence
    per channel whose decay and input gate come from block-diagonal products."""
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = time_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = torch.sigmoid(block_diagonal(u, w[p + "ra"], w[p + "ra.b"]))
    i = torch.sigmoid(block_diagonal(u, w[p + "ri"], w[p + "ri.b"]))
    lam = w[p + "lam"]
    log_a = -8.0 * r * (torch.log1p(torch.exp(-lam.abs())) + torch.clamp(lam, min=0.0))
    s = torch.zeros_like(u[0])
    rows = []
    for t in range(h.shape[0]):
        s = torch.exp(log_a[t]) * s + torch.sqrt(-torch.expm1(2.0 * log_a[t])) * i[t] * u[t]
        rows.append(s)
    return (torch.stack(rows) * y) @ w[p + "o"].T


def gla(w, p, h, m, eps):
    """Gated linear attention: a matrix state per head whose key rows decay each by a factor of their own."""
    t, nh, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(t, nh, d) * d ** -0.5
    k = (h @ w[p + "k"].T).reshape(t, nh, d)
    v = (h @ w[p + "v"].T).reshape(t, nh, dv)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    alpha = (torch.sigmoid(z) ** (1.0 / m["tau"])).reshape(t, nh, d)
    out = torch.zeros((t, nh, dv), dtype=F)
    for a in range(nh):
        s = torch.zeros((d, dv), dtype=F)
        for i in range(t):
            s = alpha[i, a].reshape(-1, 1) * s + torch.outer(k[i, a], v[i, a])
            out[i, a] = s.T @ q[i, a]
    out = unit_rms(out, eps) * w[p + "norm"]
    return (out.reshape(t, nh * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- the layer and the model ------------------------------------------------------------------------
def mlp(w, p, h):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def scalar_norm(x, g, eps):
    return unit_rms(x, eps) * g


def gated(w, name, h, y):
    """A sublayer's result times ``sigmoid(W h + b)``, element by element."""
    return y * torch.sigmoid(h @ w[name].T + w[name + ".b"])


def mixer(cfg, w, i, h, v_first=None):
    """Output of layer i's mixer for rows ``h`` and, for attention, its own values (else None)."""
    entry, p, eps = cfg["layers"][i], f"l{i}.mix.", cfg["norm"]["eps"]
    if entry["type"] == "attention":
        return attention(w, p, h, entry["mixer"], eps, v_first)
    if entry["type"] == "rglru":
        return rglru(w, p, h, entry["mixer"]), None
    return gla(w, p, h, entry["mixer"], eps), None


def layer(cfg, w, i, x, kept):
    """``kept["v"]``: the values of the first layer that mixes values, once that layer has run."""
    entry, p, eps, m = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"], cfg["residual_mult"]
    h = scalar_norm(x, w[p + "norm1"], eps)
    mixes = entry["type"] == "attention" and bool(entry["mixer"].get("v_mix"))
    y, own = mixer(cfg, w, i, token_shift(h, w[p + "shift"]), kept.get("v") if mixes else None)
    if mixes:
        kept.setdefault("v", own)
    x = x + m * gated(w, p + "rg1", h, y)
    if entry.get("mlp") is not None:
        h = scalar_norm(x, w[p + "norm2"], eps)
        x = x + m * gated(w, p + "rg2", h, mlp(w, p + "mlp.", h))
    return x


def forward(cfg, w, tokens, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` (a list) receives the rows behind every layer."""
    x, kept = embed(cfg, w, tokens), {}
    for i in range(len(cfg["layers"])):
        x = layer(cfg, w, i, x, kept)
        if layers_out is not None:
            layers_out.append(x)
    return scalar_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T * cfg["logit_scale"]


def greedy(cfg, w, prompt, n):
    """``n`` tokens by argmax, each from a whole pass over everything so far."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(torch.argmax(forward(cfg, w, tokens)[-1])))
    return tokens[len(prompt):]
