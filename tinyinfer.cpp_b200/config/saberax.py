"""Typed configuration of the Saberax decoder and its plan.

``config.json`` of this design is nested: ``architecture`` (the string ``Saberax``), ``vocab``,
``width``, ``norm.eps``, ``residual_mult`` and ``layers``, a list with one object per layer: ``type``
(the mixer's kind), ``mixer`` (its sizes and constants), ``mlp`` (the feed-forward, or null) and, for a
layer that uses another layer's tensors, ``weights_of``.  Sizes and constants have no defaults; groups
of experts and a shared expert that are not named do not exist.

The layer (``parts/block.py``, ``scaled_prenorm``): ``x += m mixer(norm1(x))`` then, where the layer has a
feed-forward, ``x += m ff(norm2(x))``, with ``m`` the ``residual_mult`` and layer norms with weight and bias.
Mixers:

``attention``   grouped-query attention inside chunks of ``mask.size`` positions whose values are the
                projected keys, a half-split turn with frequencies scaled by wavelength, unit heads behind
                the turn, a sink per head and a gate per head (``parts/chunked_attention.py``)
``parallel``    two mixers side by side (``parts/parallel_mixers.py``), their outputs normed and halved: on
                the left causal attention without a turn, heads normed with a weight and queries times a
                factor of their position (``q_temp``); on the right a gated linear recurrence per channel
                (``parts/gated_linear.py``)
``parallel_2``  the same frame: on the left attention in a window of ``mask.size`` tokens with biases, a turn
                of neighbouring pairs with stretched frequencies and unit heads behind it; on the right gated
                linear attention (``parts/state_mixers.py``)

The feed-forward is dense, gated by silu (``parts/mlp.py``), or routed experts without a gate, ``Wdown
relu(Wup h)^2``, chosen by a sigmoid router with a correction, groups valued by their two largest choice
scores, and weights brought to the sum ``router.scale`` (``parts/moe.py``).  The head has a table of its own
behind ``final.norm``.

Tensor names: ``embed``, ``head``, ``final.norm``, ``l<i>.norm1``, ``l<i>.norm2`` (each norm with ``.b``),
``l<i>.mix.*`` (attention: ``q k sink g o``; parallel: ``left.{q,k,v,q.norm,k.norm,o}``, ``right.{y,y.b,x,x.b,
conv,conv.b,ra,ra.b,ri,ri.b,lam,o}``; parallel_2: ``left.{q,q.b,k,k.b,v,v.b,o}``, ``right.{q,k,v,g,a1,a2,a2.b,
norm,o}``; both: ``left.out``, ``right.out``), ``l<i>.mlp.{gate,up,down}`` or ``l<i>.mlp.{router, correction,
e<n>.up, e<n>.down, shared.up, shared.down}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional

from .kagorax import MAX_POSITION, _get, _int, _positive
from .plan import LayerPlan, ModelPlan, PartSpec, ScheduleEntry
from .registry import Architecture, ConfigError, register_architecture
from .vametar import DECAY_POWER, _number

MIXER_TYPES = ("attention", "parallel", "parallel_2")
SIDE_SCALE = 0.5             # the design's constant on each of two mixers side by side


def _heads(entry, where: str, path: str) -> dict:
    out = {"heads": _int(entry, path + ".heads"), "kv_heads": _int(entry, path + ".kv_heads"),
           "dim": _int(entry, path + ".dim"), "vdim": _int(entry, path + ".vdim"), "scale": _number(entry, path + ".scale")}
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"'{where}.{path}': {out['heads']} heads cannot share {out['kv_heads']} kv heads evenly")
    return out


def _rotation(entry, where: str, path: str, dim: int, names: tuple[str, ...]) -> dict:
    """``rot``: how much of a head is turned, its base, and the constants ``names`` of its scaling."""
    dims = _int(entry, path + ".rot.dims", 0)
    if dims % 2 or dims > dim:
        raise ConfigError(f"'{where}.{path}.rot.dims' must be even and at most {dim}, got {dims}")
    if dims == 0:
        return {"dims": 0}
    out = {"dims": dims, "base": _positive(entry, path + ".rot.base"), "scaling": None}
    if _get(entry, path + ".rot").get("scaling") is not None:
        out["scaling"] = {n: _positive(entry, f"{path}.rot.scaling.{n}") for n in names}
    return out


def _mixer(entry, where: str, kind: str) -> dict:
    if not isinstance(entry.get("mixer"), Mapping):
        raise ConfigError(f"'{where}.mixer' must be an object")
    if kind == "attention":
        out = _heads(entry, where, "mixer")
        if out["vdim"] != out["dim"]:
            raise ConfigError(f"'{where}.mixer.vdim' is {out['vdim']}, but the values are the keys of {out['dim']} elements")
        out["chunk"] = _int(entry, "mixer.mask.size")
        out["rot"] = _rotation(entry, where, "mixer", out["dim"], ("factor", "original", "low", "high"))
        return out
    left = _heads(entry, where, "mixer.left")
    if kind == "parallel":
        left["q_temp"] = (_number(entry, "mixer.left.q_temp.coef"), _int(entry, "mixer.left.q_temp.every"))
        right = {n: _int(entry, "mixer.right." + n) for n in ("width", "blocks", "conv")}
        if right["width"] % right["blocks"]:
            raise ConfigError(f"'{where}.mixer.right': a width of {right['width']} does not fall into {right['blocks']} "
                              f"equal blocks")
    else:
        left["window"] = _int(entry, "mixer.left.mask.size")
        left["rot"] = _rotation(entry, where, "mixer.left", left["dim"], ("factor", "original", "fast", "slow"))
        right = {n: _int(entry, "mixer.right." + n) for n in ("heads", "dim", "vdim")}
        right["tau"] = _positive(entry, "mixer.right.tau")
        # inner width of the decay's two products: the stored tensors' own; a configuration names it
        # only for random weights
        rank = _get(entry, "mixer.right").get("decay_rank")
        right["decay_rank"] = None if rank is None else _int(entry, "mixer.right.decay_rank")
    return {"left": left, "right": right}


def _mlp(entry, where: str) -> Optional[dict]:
    mlp = entry.get("mlp")
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, Mapping) else mlp
    if kind == "dense":
        return {"kind": "dense", "ff": _int(mlp, "ff")}
    if kind != "moe":
        raise ConfigError(f"'{where}.mlp.kind' is {kind!r}; known: 'dense', 'moe'")
    experts, top = _int(mlp, "router.experts"), _int(mlp, "router.top")
    groups = None
    if _get(mlp, "router").get("groups") is not None:
        groups = (_int(mlp, "router.groups.count"), _int(mlp, "router.groups.keep"))
    count, keep = groups or (1, 1)
    if experts % count or keep > count:
        raise ConfigError(f"'{where}.mlp.router': {experts} experts do not fall into {count} equal groups of which {keep} "
                          f"are kept")
    if top > experts // count * keep:
        raise ConfigError(f"'{where}.mlp.router': top {top} of {experts // count * keep} experts")
    shared = None if mlp.get("shared") is None else {"ff": _int(mlp, "shared.ff")}
    return {"kind": "moe", "experts": experts, "top": top, "groups": groups, "scale": _number(mlp, "router.scale"),
            "ff": _int(mlp, "expert.ff"), "shared": shared}


@dataclass(frozen=True)
class SaberaxLayer:
    type: str
    mixer: Mapping[str, Any]            # the validated sizes and constants of the mixer
    mlp: Optional[Mapping[str, Any]]    # None: no feed-forward
    weights_of: Optional[int] = None    # the layer whose tensors this one uses (None: its own)


@dataclass(frozen=True)
class SaberaxConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: tuple[SaberaxLayer, ...]
    source: Mapping[str, Any]

    ARCHITECTURE = "Saberax"

    @staticmethod
    def from_dict(cfg: Mapping[str, Any]) -> "SaberaxConfig":
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
            owner = entry.get("weights_of")
            if owner is not None and (isinstance(owner, bool) or not isinstance(owner, int)
                                      or not 0 <= owner < len(raw) or owner == i):
                raise ConfigError(f"'{where}.weights_of' must name another layer, got {owner!r}")
            layers.append(SaberaxLayer(kind, _mixer(entry, where, kind), _mlp(entry, where), owner))
        out = SaberaxConfig(vocab=vocab, width=width, norm_eps=_positive(cfg, "norm.eps"),
                            residual_mult=_number(cfg, "residual_mult"), layers=tuple(layers), source=dict(cfg))
        for i, layer in enumerate(layers):
            src = layers[out.owner(i)]
            if (src.type, src.mixer, src.mlp) != (layer.type, layer.mixer, layer.mlp):
                raise ConfigError(f"'layers[{i}]' uses layer {layer.weights_of}'s tensors but its type, sizes or constants "
                                  f"differ")
        return out

    def owner(self, i: int) -> int:
        """The layer that owns the tensors of layer ``i``."""
        seen = {i}
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
            if i in seen:
                raise ConfigError(f"'layers[{i}].weights_of' leads back to itself: no layer owns the tensors")
            seen.add(i)
        return i

    def to_dict(self) -> dict[str, Any]:
        return dict(self.source)


def _position(m: Mapping[str, Any], kind: str, scaled: str, layout: str) -> PartSpec:
    rot = m["rot"]
    if not rot["dims"]:
        return PartSpec("none", {"head_dim": m["dim"]})
    base = {"head_dim": m["dim"], "theta": rot["base"], "rotary_dim": rot["dims"]}
    if rot["scaling"] is None:
        return PartSpec(kind, base)
    return PartSpec(scaled, {**base, **rot["scaling"], "layout": layout})


def _attention_spec(cfg: SaberaxConfig, m: Mapping[str, Any], position: PartSpec, **options: Any) -> PartSpec:
    return PartSpec("chunked_attention", {
        "hidden_size": cfg.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
        "v_head_dim": m["vdim"], "scale": m["scale"], "qk_norm_eps": cfg.norm_eps, "position": position,
        "norm_per_head": True, "head_temperature": False, "head_gate": False, **options})


def _mixer_spec(cfg: SaberaxConfig, layer: SaberaxLayer) -> PartSpec:
    m = layer.mixer
    if layer.type == "attention":
        options = {"norm_before": False, "norm_after": True, "values_from_keys": True, "sink": True, "head_gate": True,
                   "chunk": m["chunk"]}
        return _attention_spec(cfg, m, _position(m, "rope_neox", "rope_wavelength", "neox"), **options)
    a, b = m["left"], m["right"]
    if layer.type == "parallel":
        left = _attention_spec(cfg, a, PartSpec("none", {"head_dim": a["dim"]}), query_factor=a["q_temp"])
        right = PartSpec("gated_linear_recurrence", {
            "hidden_size": cfg.width, "width": b["width"], "blocks": b["blocks"], "conv_taps": b["conv"],
            "decay_power": DECAY_POWER})
    else:
        left = _attention_spec(cfg, a, _position(a, "rope_interleaved", "rope_stretched", "interleaved"),
                               norm_before=False, norm_after=True, bias=True, window=a["window"])
        right = PartSpec("gated_linear_attention", {
            "hidden_size": cfg.width, "num_heads": b["heads"], "head_dim": b["dim"], "v_head_dim": b["vdim"],
            "tau": b["tau"], "norm_eps": cfg.norm_eps, "decay_rank": b["decay_rank"]})
    return PartSpec("parallel_mixers", {"hidden_size": cfg.width, "left": left, "right": right, "left_scale": SIDE_SCALE,
                                        "right_scale": SIDE_SCALE, "norm_eps": cfg.norm_eps})


def _ffn_spec(cfg: SaberaxConfig, mlp: Mapping[str, Any]) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("glu_mlp", {"hidden_size": cfg.width, "intermediate_size": mlp["ff"], "activation": "silu"})
    shared = mlp["shared"]
    return PartSpec("routed_experts", {
        "hidden_size": cfg.width, "experts": mlp["experts"], "top": mlp["top"], "expert_size": mlp["ff"],
        "router": "sigmoid", "activation": ("relu2", 0.0, 0.0), "correction": True, "groups": mlp["groups"],
        "group_score": "top2", "normalize": True, "weight_scale": mlp["scale"],
        "shared_size": None if shared is None else shared["ff"], "shared_gated": False})


def build_plan(cfg: SaberaxConfig) -> ModelPlan:
    def norm(tensor: str) -> PartSpec:
        return PartSpec("layer_norm", {"size": cfg.width, "eps": cfg.norm_eps, "tensor": tensor})

    # the plan's layers are the layers that own tensors; the schedule runs one entry per layer of
    # the configuration, each with a cache slot of its own
    index_of: dict[int, int] = {}
    layers = []
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of is not None:
            continue
        index_of[i] = len(layers)
        p = f"l{i}."
        has_ff = layer.mlp is not None
        layers.append(LayerPlan(
            block=PartSpec("scaled_prenorm", {"multiplier": cfg.residual_mult}), mixer=_mixer_spec(cfg, layer),
            ffn=_ffn_spec(cfg, layer.mlp) if has_ff else None,
            mixer_norm=norm("norm1"), ffn_norm=norm("norm2") if has_ff else None,
            names={"mixer": p + "mix.", "ffn": p + "mlp.", "mixer_norm": p, "ffn_norm": p}))
    schedule = [ScheduleEntry(layer=index_of[cfg.owner(i)], cache_slot=i) for i in range(len(cfg.layers))]
    return ModelPlan(
        architecture=cfg.ARCHITECTURE, hidden_size=cfg.width, vocab_size=cfg.vocab, max_position=MAX_POSITION,
        layers=layers, schedule=schedule,
        embedding=PartSpec("embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tensor": "embed"}),
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied": False, "tensor": "head"}),
        names={"embedding": "", "final_norm": "", "head": ""})


register_architecture(Architecture(
    name=SaberaxConfig.ARCHITECTURE, from_dict=SaberaxConfig.from_dict, build_plan=build_plan,
    aliases=("saberax",)))
