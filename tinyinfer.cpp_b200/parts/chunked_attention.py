"""Grouped-query attention inside chunks of positions, with a norm over the whole query and key
rows, a score factor per head, a cap on the score and an output gate per head.

For token ``i`` and query head ``a`` (kv head ``a // (heads / kv_heads)``):

* ``q, k, v = Wq h, Wk h, Wv h`` (no biases); ``q`` (all heads as one row) and ``k`` likewise are
  RMS-normed with a weight per column, then the first ``rotary_dim`` elements of every head are
  turned by the position part's rule.
* key ``j <= i`` is visible when ``j // chunk == i // chunk`` (chunks are counted from the
  sequence's position 0) and, if a window is given, ``i - j < window``.
* ``score = (q . k) * scale * temp[a]``, then ``softcap * tanh(score / softcap)``; float32 softmax
  over the visible keys; weighted sum of the values (head size ``v_head_dim``).
* head ``a``'s output times ``sigmoid((Wg h)[a])``, then ``residual += Wo (.)``.

``Wq, Wk, Wv, Wg`` run as one product.  Every option can be left out (``chunk``, ``window``,
``softcap`` None; ``head_temperature``, ``head_gate`` False), and ``norm_per_head`` norms every
query and key head by itself with one weight of ``head_dim`` elements, so other designs can use the
part: with everything off it is plain causal grouped-query attention with a query/key norm.

More options, for heads that are prepared one by one (``heads_prepare_store``): ``norm_before`` False leaves the
norm in front of the turn out (no ``q.norm``, ``k.norm``); ``norm_after`` divides every query and key head by its
root mean square behind the turn; ``bias`` adds a stored bias to q, k and v (``q.b`` ...); ``query_factor = (coef,
every)`` multiplies the query at position ``p`` by ``1 + coef ln(floor((p + 1) / every) + 1)``; ``values_from_keys``
takes the projected keys, before norm and turn, as values (no ``v``); ``sink`` adds ``exp(sink[a])`` to the
softmax's denominator (a number per head, without a key or a value).

``value_mix`` ties the values of several layers together: the layer with ``"source"`` leaves its values
``v1`` (float32, in the step's scratch), and a later layer with ``"mix"`` caches ``(1 - l) v + l v1`` of
the same token (``l`` the number in the tensor ``vmix``).
"""
from __future__ import annotations

from typing import Optional

import torch

from ..config.plan import PartSpec
from .base import (MATRIX, NORM_WEIGHT, NORM_ZERO, PagedKVSpec, ProjectedMixer, WeightSpec, as_float32, build_part,
                   register_part, stack_rows)


class ChunkedAttention(ProjectedMixer):
    defers = True

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, v_head_dim: int,
                 scale: float, qk_norm_eps: float, position: PartSpec, chunk: Optional[int] = None,
                 window: Optional[int] = None, softcap: Optional[float] = None,
                 head_temperature: bool = True, head_gate: bool = True, norm_per_head: bool = False,
                 value_mix: Optional[str] = None, norm_before: bool = True, norm_after: bool = False, bias: bool = False,
                 query_factor=None, values_from_keys: bool = False, sink: bool = False):
        if value_mix not in (None, "source", "mix"):
            raise ValueError(f"value_mix must be None, 'source' or 'mix', got {value_mix!r}")
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} heads cannot share {num_kv_heads} kv heads evenly")
        for name, v in (("chunk", chunk), ("window", window)):
            if v is not None and v < 1:
                raise ValueError(f"{name} must be positive, got {v}")
        self.hidden_size = int(hidden_size)
        self.num_heads, self.num_kv_heads = int(num_heads), int(num_kv_heads)
        self.head_dim, self.v_head_dim = int(head_dim), int(v_head_dim)
        self.scale, self.eps = float(scale), float(qk_norm_eps)
        self.chunk = None if chunk is None else int(chunk)
        self.window = None if window is None else int(window)
        self.softcap = None if softcap is None else float(softcap)
        self.head_temperature, self.head_gate = bool(head_temperature), bool(head_gate)
        # the norm of queries and keys: over the whole row with a weight per column, or over each
        # head by itself with a weight of head_dim elements that all heads share
        self.norm_per_head = bool(norm_per_head)
        if self.norm_per_head and value_mix is not None:
            raise ValueError("values are mixed beside a norm over whole rows only")
        self.norm_before, self.norm_after, self.has_bias = bool(norm_before), bool(norm_after), bool(bias)
        self.query_factor = None if query_factor is None else (float(query_factor[0]), int(query_factor[1]))
        self.values_from_keys, self.has_sink = bool(values_from_keys), bool(sink)
        # heads one by one, with whatever of these options there is
        self.by_heads = (not self.norm_before or self.norm_after or self.has_bias or self.query_factor is not None
                         or self.values_from_keys)
        if self.by_heads and (value_mix is not None or (self.norm_before and not self.norm_per_head)):
            raise ValueError("heads that are prepared one by one have norms per head and values of their own")
        if self.values_from_keys and head_dim != v_head_dim:
            raise ValueError(f"values of {v_head_dim} elements cannot be keys of {head_dim}")
        if self.query_factor is not None and self.query_factor[1] < 1:
            raise ValueError(f"the query's factor grows every {query_factor[1]} positions; that must be positive")
        self.position = build_part("position", position)
        self.value_mix, self.mix_share = value_mix, 0.0
        self.nq, self.nk = self.num_heads * self.head_dim, self.num_kv_heads * self.head_dim
        self.nv = 0 if self.values_from_keys else self.num_kv_heads * self.v_head_dim
        self.no = self.num_heads * self.v_head_dim
        self.projected = ("q", "k") if self.values_from_keys else ("q", "k", "v")
        self.q_norm = self.k_norm = self.temp = self.sink = self.bias = None

    def weight_specs(self):
        h = self.hidden_size
        rows = {"q": self.nq, "k": self.nk, "v": self.nv}
        specs = {"o": WeightSpec((h, self.no), MATRIX)}
        for name in self.projected:
            specs[name] = WeightSpec((rows[name], h), MATRIX)
            if self.has_bias:
                specs[name + ".b"] = WeightSpec((rows[name],), NORM_ZERO)
        if self.norm_before:
            specs["q.norm"] = WeightSpec((self.head_dim if self.norm_per_head else self.nq,), NORM_WEIGHT)
            specs["k.norm"] = WeightSpec((self.head_dim if self.norm_per_head else self.nk,), NORM_WEIGHT)
        if self.has_sink:
            specs["sink"] = WeightSpec((self.num_heads,), NORM_ZERO)
        if self.value_mix is not None:                # the source may store a number that it does not use
            specs["vmix"] = WeightSpec((), NORM_ZERO, optional=self.value_mix == "source")
        if self.head_temperature:
            specs["temp"] = WeightSpec((self.num_heads,), NORM_WEIGHT)
        if self.head_gate:
            specs["g"] = WeightSpec((self.num_heads, h), MATRIX)
        return specs

    def load_weights(self, tensors, ops):
        mats = [tensors[n] for n in self.projected + (("g",) if self.head_gate else ())]
        self.w_in = ops.pack_linear(stack_rows(mats, self.hidden_size))
        self.w_o = ops.pack_linear(tensors["o"])
        if self.norm_before:
            self.q_norm = as_float32(tensors["q.norm"]).contiguous()
            self.k_norm = as_float32(tensors["k.norm"]).contiguous()
        if self.has_bias:
            self.bias = torch.cat([as_float32(tensors[n + ".b"]) for n in self.projected]).contiguous()
        self.sink = as_float32(tensors["sink"]).contiguous() if self.has_sink else None
        self.temp = as_float32(tensors["temp"]).contiguous() if self.head_temperature else None
        if self.value_mix == "mix":                   # a constant of the model
            self.mix_share = float(as_float32(tensors["vmix"]).reshape(()).item())
        if hasattr(ops, "want_row_tiles"):
            ops.want_row_tiles(self.num_heads, self.num_kv_heads)

    def cache_spec(self):
        return PagedKVSpec(self.num_kv_heads, self.head_dim, self.window,
                           None if self.v_head_dim == self.head_dim else self.v_head_dim, 0, self.chunk)

    def mix(self, ops, proj, step, cache, dtype):
        t, dev = proj.shape[0], proj.device
        q = torch.empty((t, self.nq), dtype=dtype, device=dev)
        rotation = self.position.rotation(dev)
        if self.value_mix == "source":
            step.scratch["value_mix"] = proj[:, self.nq + self.nk:self.nq + self.nk + self.nv]
        if self.by_heads:
            ops.heads_prepare_store(proj, rotation, step, cache, q, self.num_heads, self.num_kv_heads, self.head_dim,
                                    self.v_head_dim, bias=self.bias,
                                    pre_norm=(self.q_norm, self.k_norm, self.eps) if self.norm_before else None,
                                    post_norm_eps=self.eps if self.norm_after else None, query_factor=self.query_factor,
                                    values_from_keys=self.values_from_keys)
        elif rotation.kind == "neox" or self.value_mix is not None:
            mixed = (step.scratch["value_mix"], self.mix_share) if self.value_mix == "mix" else None
            ops.qkv_turn_store(proj, rotation, None, step, cache, q, self.num_heads, self.num_kv_heads, self.head_dim,
                               self.v_head_dim, row_norm=(self.q_norm, self.k_norm, self.eps), value_mix=mixed)
        else:
            ops.qk_rownorm_rope_store(proj, self.q_norm, self.k_norm, self.eps, rotation, step, cache, q,
                                      self.num_heads, self.num_kv_heads, self.head_dim, self.v_head_dim,
                                      per_head=self.norm_per_head)
        at_g = self.nq + self.nk + self.nv
        gate = proj[:, at_g:at_g + self.num_heads] if self.head_gate else None
        out = torch.empty((t, self.no), dtype=dtype, device=dev)
        ops.attention_options(q, step, cache, out, self.num_heads, self.num_kv_heads, self.head_dim,
                              self.v_head_dim, self.scale, window=self.window, chunk=self.chunk,
                              softcap=self.softcap, head_scale=self.temp, sink=self.sink, gate=gate, gate_per_head=True)
        return out


register_part("mixer", "chunked_attention", ChunkedAttention)
