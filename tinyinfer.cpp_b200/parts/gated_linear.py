"""A recurrent mixer with a vector state: a linear recurrence per channel under gates (the recurrent
block of Griffin with its real-gated linear recurrent unit).

Two branches of ``width`` channels from the mixer's input ``h``:

    y = gelu(Wy h + by)                               (the tanh form of gelu)
    u_t = b + sum_j c[:, j] (Wx h + bx)_(t - taps + 1 + j)      (zeros before the sequence's start)

``u`` falls into ``blocks`` equal parts; in part ``b``, ``r = sigmoid(Ra[b] u_b + ra[b])`` and ``i =
sigmoid(Ri[b] u_b + ri[b])`` with square matrices.  With ``log a = -decay_power * r * softplus(lam)``
per channel and ``S = 0`` at the start

    S <- a S + sqrt(1 - a^2) i u;        residual += Wo (S * y)

``Wy`` and ``Wx`` run as one product, ``Ra`` and ``Ri`` as one product per part.  ``u``, both gates, the
decay and the state are float32 whatever the activation dtype.  Per request the slot keeps the state
and the convolution's last ``taps - 1`` inputs (with their bias).
"""
from __future__ import annotations

import torch

from .base import MATRIX, NORM_ZERO, FixedStateSpec, ProjectedMixer, WeightSpec, as_float32, register_part, stack_rows


class GatedLinearRecurrence(ProjectedMixer):
    def __init__(self, hidden_size: int, width: int, blocks: int, conv_taps: int, decay_power: float = 8.0):
        self.hidden_size, self.width, self.blocks = int(hidden_size), int(width), int(blocks)
        self.conv_taps, self.decay_power = int(conv_taps), float(decay_power)
        if self.blocks < 1 or self.width % self.blocks:
            raise ValueError(f"{self.width} channels do not fall into {self.blocks} equal blocks")
        if self.conv_taps < 1:
            raise ValueError(f"the short convolution needs at least one tap, got {conv_taps}")
        self.w_gates = self.conv_w = self.conv_b = None
        self.y_bias = self.x_bias = self.gate_bias = self.log_decay = None

    def weight_specs(self):
        n, h, b = self.width, self.hidden_size, self.blocks
        per = n // b
        return {"y": WeightSpec((n, h), MATRIX), "y.b": WeightSpec((n,), NORM_ZERO),
                "x": WeightSpec((n, h), MATRIX), "x.b": WeightSpec((n,), NORM_ZERO),
                "conv": WeightSpec((n, self.conv_taps), MATRIX), "conv.b": WeightSpec((n,), NORM_ZERO),
                "ra": WeightSpec((b, per, per), MATRIX), "ra.b": WeightSpec((b, per), NORM_ZERO),
                "ri": WeightSpec((b, per, per), MATRIX), "ri.b": WeightSpec((b, per), NORM_ZERO),
                "lam": WeightSpec((n,), NORM_ZERO), "o": WeightSpec((h, n), MATRIX)}

    def load_weights(self, tensors, ops):
        self.w_in = ops.pack_linear(stack_rows([tensors["y"], tensors["x"]], self.hidden_size))
        self.w_o = ops.pack_linear(tensors["o"])
        ra, ri = tensors["ra"], tensors["ri"]
        if ra.dtype != ri.dtype:                      # mixed storage: widen, never narrow
            ra, ri = ra.to(torch.float32), ri.to(torch.float32)
        self.w_gates = ops.pack_block_gates(ra, ri)
        vec = lambda name: as_float32(tensors[name]).reshape(-1).contiguous()
        self.conv_w = as_float32(tensors["conv"]).contiguous()
        self.conv_b, self.x_bias, self.y_bias = vec("conv.b"), vec("x.b"), vec("y.b")
        self.gate_bias = torch.stack([vec("ra.b"), vec("ri.b")]).contiguous()
        # log a per unit of the gate r, made once in double precision
        lam = tensors["lam"].to(torch.float64)
        self.log_decay = (-self.decay_power * torch.nn.functional.softplus(lam)).to(torch.float32).contiguous()

    def cache_spec(self):
        return FixedStateSpec((self.width * self.conv_taps,), torch.float32)      # the state, taps - 1 rows

    def mix(self, ops, proj, step, cache, dtype):
        t, dev, n = proj.shape[0], proj.device, self.width
        u = torch.empty((t, n), dtype=torch.float32, device=dev)
        ops.causal_conv(proj[:, n:2 * n], self.conv_w, step, cache, n, u, renew=True, in_bias=self.x_bias, bias=self.conv_b)
        out = torch.empty((t, n), dtype=dtype, device=dev)
        ops.gated_recurrence(u, self.w_gates, self.gate_bias, self.log_decay, proj[:, :n], self.y_bias, step, cache, out)
        return out


register_part("mixer", "gated_linear_recurrence", GatedLinearRecurrence)
