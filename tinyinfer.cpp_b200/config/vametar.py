"""Typed configuration of the Vametar decoder and its plan.

``config.json`` of this design is nested: ``architecture`` (the string ``Vametar``), ``vocab``,
``width``, ``embedding.bigram``, ``norm.eps``, ``residual_mult``, ``logit_scale`` and ``layers``, a
list with one object per layer: ``type`` (the mixer's kind), ``mixer`` (its sizes and constants) and
``mlp`` (the feed-forward, or null).  Nothing has a default.

The layer (``parts/block.py``, ``gated_prenorm``): with ``h = norm1(x)``, ``x += m sigmoid(Wg1 h +
bg1) * mixer(h + (h' - h) shift)``, then, where the layer has a feed-forward, the same with
``norm2``, ``Wg2`` and no shift; ``m`` is ``residual_mult`` and ``h'`` the row of the token before.
Every norm is an RMS norm whose weight is one number.  Mixers:

``attention``  grouped-query attention, causal, with an RMS norm over the whole query row and the
               whole key row, a half-split turn of the first ``rot.dims`` elements of a head, and
               values mixed with those of the first layer that has ``v_mix``
               (``parts/chunked_attention.py``)
``rglru``      two branches of ``width``: a gelu, and a short convolution over time in front of a
               linear recurrence per channel with block-diagonal gates (``parts/gated_linear.py``)
``gla``        gated linear attention, a matrix state per head with a decay per key channel
               (``parts/state_mixers.py``)

The feed-forward is gated by a gelu (``parts/mlp.py``).  The embedding adds a row of a second table
that a hash of the last two tokens chooses (``parts/embed_head.py``).  The head has a table of its
own behind ``final.norm``; ``logit_scale`` multiplies the logits (as a factor on the normed row).

Tensor names: ``embed``, ``bigram``, ``head``, ``final.norm``, ``l<i>.{norm1,norm2}``, ``l<i>.shift``,
``l<i>.{rg1,rg1.b,rg2,rg2.b}``, ``l<i>.mix.*`` (attention: ``q k v q.norm k.norm vmix o``; rglru: ``y y.b
x x.b conv conv.b ra ra.b ri ri.b lam o``; gla: ``q k v g a1 a2 a2.b norm o``), ``l<i>.mlp.{gate,up,down}``.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Mapping, Optional

from .kagorax import MAX_POSITION, _get, _int, _positive
from .plan import LayerPlan, ModelPlan, PartSpec, default_schedule
from .registry import Architecture, ConfigError, register_architecture

MIXER_TYPES = ("attention", "rglru", "gla")
DECAY_POWER = 8.0            # the design's constant in front of the recurrence gate: log a = -8 r softplus(lam)


def _number(cfg, path: str) -> float:
    v = _get(cfg, path)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(v):
        raise ConfigError(f"'{path}' must be a finite number, got {v!r}")
    return float(v)


def _whole(cfg, path: str) -> int:
    v = _get(cfg, path)
    if isinstance(v, bool) or not isinstance(v, int):
        raise ConfigError(f"'{path}' must be an integer, got {v!r}")
    return v


def _mixer(entry, where: str, kind: str) -> dict:
    if not isinstance(entry.get("mixer"), Mapping):
        raise ConfigError(f"'{where}.mixer' must be an object")
    if kind == "rglru":
        out = {"width": _int(entry, "mixer.width"), "blocks": _int(entry, "mixer.blocks"), "conv": _int(entry, "mixer.conv")}
        if out["width"] % out["blocks"]:
            raise ConfigError(f"'{where}.mixer': a width of {out['width']} does not fall into {out['blocks']} equal blocks")
        return out
    out = {"heads": _int(entry, "mixer.heads"), "dim": _int(entry, "mixer.dim"), "vdim": _int(entry, "mixer.vdim")}
    if kind == "gla":
        out["tau"] = _positive(entry, "mixer.tau")
        # inner width of the decay's two products: the stored tensors' own; a configuration names it
        # only for random weights
        rank = entry["mixer"].get("decay_rank")
        out["decay_rank"] = None if rank is None else _int(entry, "mixer.decay_rank")
        return out
    out.update(kv_heads=_int(entry, "mixer.kv_heads"), scale=_number(entry, "mixer.scale"),
               rot_dims=_int(entry, "mixer.rot.dims", 0), v_mix=bool(entry["mixer"].get("v_mix", False)))
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"'{where}.mixer': {out['heads']} heads cannot share {out['kv_heads']} kv heads evenly")
    if out["rot_dims"] % 2 or out["rot_dims"] > out["dim"]:
        raise ConfigError(f"'{where}.mixer.rot.dims' must be even and at most {out['dim']}, got {out['rot_dims']}")
    out["rot_base"] = _positive(entry, "mixer.rot.base") if out["rot_dims"] else 1.0
    return out


def _mlp(entry, where: str) -> Optional[dict]:
    mlp = entry.get("mlp")
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, Mapping) else mlp
    if kind != "dense":
        raise ConfigError(f"'{where}.mlp.kind' is {kind!r}; known: 'dense'")
    return {"ff": _int(mlp, "ff")}


@dataclass(frozen=True)
class VametarLayer:
    type: str
    mixer: Mapping[str, Any]            # the validated sizes and constants of the mixer
    mlp: Optional[Mapping[str, Any]]    # None: no feed-forward


@dataclass(frozen=True)
class VametarConfig:
    vocab: int
    width: int
    buckets: int
    mul_prev: int
    mul_cur: int
    norm_eps: float
    residual_mult: float
    logit_scale: float
    layers: tuple[VametarLayer, ...]
    source: Mapping[str, Any]

    ARCHITECTURE = "Vametar"

    @staticmethod
    def from_dict(cfg: Mapping[str, Any]) -> "VametarConfig":
        vocab, width = _int(cfg, "vocab"), _int(cfg, "width")
        raw = _get(cfg, "layers")
        if not isinstance(raw, (list, tuple)) or not raw:
            raise ConfigError("'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw):
            where = f"layers[{i}]"
            if not isinstance(entry, Mapping):
                raise ConfigError(f"'{where}' must be an object")
            kind = entry.get("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"'{where}.type' is {kind!r}; known: {', '.join(MIXER_TYPES)}")
            layers.append(VametarLayer(kind, _mixer(entry, where, kind), _mlp(entry, where)))
        mixed = [(i, la.mixer["kv_heads"] * la.mixer["vdim"]) for i, la in enumerate(layers)
                 if la.type == "attention" and la.mixer["v_mix"]]
        for i, n in mixed[1:]:
            if n != mixed[0][1]:
                raise ConfigError(f"'layers[{i}].mixer': values of {n} elements cannot be mixed with the {mixed[0][1]} "
                                  f"elements of layer {mixed[0][0]}")
        return VametarConfig(
            vocab=vocab, width=width, buckets=_int(cfg, "embedding.bigram.buckets"),
            mul_prev=_whole(cfg, "embedding.bigram.mul_prev"), mul_cur=_whole(cfg, "embedding.bigram.mul_cur"),
            norm_eps=_positive(cfg, "norm.eps"), residual_mult=_number(cfg, "residual_mult"),
            logit_scale=_number(cfg, "logit_scale"), layers=tuple(layers), source=dict(cfg))

    def to_dict(self) -> dict[str, Any]:
        return dict(self.source)


def _mixer_spec(cfg: VametarConfig, layer: VametarLayer, value_mix: Optional[str] = None) -> PartSpec:
    """``value_mix``: None, ``"source"`` (the first layer that mixes values) or ``"mix"`` (a later one)."""
    m = layer.mixer
    if layer.type == "rglru":
        return PartSpec("gated_linear_recurrence", {
            "hidden_size": cfg.width, "width": m["width"], "blocks": m["blocks"], "conv_taps": m["conv"],
            "decay_power": DECAY_POWER})
    if layer.type == "gla":
        return PartSpec("gated_linear_attention", {
            "hidden_size": cfg.width, "num_heads": m["heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
            "tau": m["tau"], "norm_eps": cfg.norm_eps, "decay_rank": m["decay_rank"]})
    position = (PartSpec("rope_neox", {"head_dim": m["dim"], "theta": m["rot_base"], "rotary_dim": m["rot_dims"]})
                if m["rot_dims"] else PartSpec("none", {"head_dim": m["dim"]}))
    return PartSpec("chunked_attention", {
        "hidden_size": cfg.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
        "v_head_dim": m["vdim"], "scale": m["scale"], "qk_norm_eps": cfg.norm_eps, "position": position,
        "head_temperature": False, "head_gate": False, "value_mix": value_mix})


def build_plan(cfg: VametarConfig) -> ModelPlan:
    def norm(tensor: str, factor: float = 1.0) -> PartSpec:
        return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "tensor": tensor, "scalar": True,
                                    "factor": factor})

    layers, source_seen = [], False
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        has_ff = layer.mlp is not None
        value_mix = None
        if layer.type == "attention" and layer.mixer["v_mix"]:
            value_mix = "mix" if source_seen else "source"
            source_seen = True
        layers.append(LayerPlan(
            block=PartSpec("gated_prenorm", {"hidden_size": cfg.width, "multiplier": cfg.residual_mult}),
            mixer=_mixer_spec(cfg, layer, value_mix),
            ffn=PartSpec("glu_mlp", {"hidden_size": cfg.width, "intermediate_size": layer.mlp["ff"],
                                     "activation": "gelu_tanh"}) if has_ff else None,
            mixer_norm=norm("norm1"), ffn_norm=norm("norm2") if has_ff else None,
            names={"block": p, "mixer": p + "mix.", "ffn": p + "mlp.", "mixer_norm": p, "ffn_norm": p}))
    return ModelPlan(
        architecture=cfg.ARCHITECTURE, hidden_size=cfg.width, vocab_size=cfg.vocab, max_position=MAX_POSITION,
        layers=layers, schedule=default_schedule(len(layers)),
        embedding=PartSpec("bigram", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "buckets": cfg.buckets,
                                      "mul_prev": cfg.mul_prev, "mul_cur": cfg.mul_cur, "tensor": "embed",
                                      "bigram_tensor": "bigram"}),
        # a factor on the rows that the head reads is the same factor on its logits
        final_norm=norm("final.norm", cfg.logit_scale),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied": False, "tensor": "head"}),
        names={"embedding": "", "final_norm": "", "head": ""})


register_architecture(Architecture(
    name=VametarConfig.ARCHITECTURE, from_dict=VametarConfig.from_dict, build_plan=build_plan,
    aliases=("vametar",)))
