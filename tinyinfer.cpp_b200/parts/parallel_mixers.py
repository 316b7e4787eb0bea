"""Two mixers side by side: both read the same input, each keeps what it needs per request, and
the layer's mixer output is ``left_scale * left(h) + right_scale * right(h)``.

With ``norm_eps`` each side's output is first RMS-normed over the model width with a weight of its
own (tensors ``left.out`` and ``right.out``): ``scale * (rms(left(h)) * wl + rms(right(h)) * wr)``, with
one ``scale`` for both sides.

The two are ordinary mixer parts (for instance causal attention beside a recurrent mixer); their
tensors live under ``left.`` and ``right.``, their caches under the same names of a composite
cache slot.  Each writes its result into float32 rows of its own, which one pass then adds,
scaled, to the output.  Where both are ``ProjectedMixer`` parts, their first products run as one over
their stacked weights, and the last two share a launch where few rows allow it.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..config.plan import PartSpec
from .base import (NORM_WEIGHT, CompositeSpec, Part, ProjectedMixer, WeightSpec, as_float32, build_part, register_part,
                   residual_and_factor, stack_rows)

SIDES = ("left", "right")


class ParallelMixers(Part):
    category = "mixer"
    takes_factor = True

    def __init__(self, hidden_size: int, left: PartSpec, right: PartSpec, left_scale: float = 1.0,
                 right_scale: float = 1.0, norm_eps: Optional[float] = None):
        self.hidden_size = int(hidden_size)
        self.sides = {"left": build_part("mixer", left), "right": build_part("mixer", right)}
        self.scales = {"left": float(left_scale), "right": float(right_scale)}
        self.norm_eps = None if norm_eps is None else float(norm_eps)
        if self.norm_eps is not None and left_scale != right_scale:
            raise ValueError("normed sides are added with one factor")
        self.out_norms = {}
        self.w_in = None                     # both sides' first products as one
        self.cut = 0                         # ... the right side's columns start here

    def weight_specs(self):
        specs = {f"{side}.{name}": spec for side in SIDES for name, spec in self.sides[side].weight_specs().items()}
        if self.norm_eps is not None:
            specs.update({f"{side}.out": WeightSpec((self.hidden_size,), NORM_WEIGHT) for side in SIDES})
        return specs

    def load_weights(self, tensors, ops):
        for side in SIDES:
            cut = side + "."
            self.sides[side].load_weights({n[len(cut):]: t for n, t in tensors.items()
                                           if n.startswith(cut) and n != cut + "out"}, ops)
            if self.norm_eps is not None:
                self.out_norms[side] = as_float32(tensors[cut + "out"]).contiguous()
        left, right = (self.sides[side] for side in SIDES)
        if isinstance(left, ProjectedMixer) and isinstance(right, ProjectedMixer) and left.w_in.shape[0] % 16 == 0:
            self.cut = left.w_in.shape[0]
            self.w_in = ops.pack_linear(stack_rows([left.w_in, right.w_in], self.hidden_size))
            left.w_in = right.w_in = None

    def step_lists(self):
        return [sl for side in SIDES for sl in self.sides[side].step_lists()]

    def cache_spec(self):
        return CompositeSpec(tuple((side, self.sides[side].cache_spec()) for side in SIDES))

    def _rows(self, ops, h, step, cache):
        """The two sides' outputs, float32 ``[2, T, width]``."""
        shape = (2, h.shape[0], self.hidden_size)
        if self.w_in is None:
            rows = torch.zeros(shape, dtype=torch.float32, device=h.device)
            for i, side in enumerate(SIDES):
                self.sides[side].forward(ops, h, rows[i], step, cache.child(side))
            return rows
        rows = torch.empty(shape, dtype=torch.float32, device=h.device)
        proj = torch.empty((h.shape[0], self.w_in.shape[0]), dtype=torch.float32, device=h.device)
        ops.linear(h, self.w_in, proj)
        parts = {"left": proj[:, :self.cut], "right": proj[:, self.cut:]}
        mixed = [self.sides[side].mix(ops, parts[side], step, cache.child(side), h.dtype) for side in SIDES]
        ops.linear(mixed[0], self.sides["left"].w_o, rows[0], may_pair=True)
        ops.linear(mixed[1], self.sides["right"].w_o, rows[1])
        return rows

    def forward(self, ops, h, residual, step, cache):
        self.forward_then(ops, h, residual, step, cache, None)

    def forward_then(self, ops, h, residual, step, cache, norm):
        """``forward``, and (``norm`` a layer norm part, or None) that norm of the new residual: in one launch with the
        sum where the sides are normed.  Returns the normed rows."""
        rows = self._rows(ops, h, step, cache)
        x, factor = residual_and_factor(residual)
        if self.norm_eps is None:
            ops.add_scaled(x, rows[0], factor * self.scales["left"], rows[1], factor * self.scales["right"])
            return None if norm is None else norm.forward(ops, x, h.dtype)
        out = None if norm is None else torch.empty_like(h)
        ops.norm_sum(rows[0], rows[1], self.out_norms["left"], self.out_norms["right"], self.norm_eps, x,
                     factor * self.scales["left"], None if norm is None else (norm.weight, norm.bias, norm.eps, out))
        return out


register_part("mixer", "parallel_mixers", ParallelMixers)
