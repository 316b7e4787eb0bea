"""Bindings of the kernels in ``csrc/matrix_state*.cu`` (library ``state``),
``csrc/channel_recurrence.cu`` (library ``channels``), ``csrc/state_rows.cu`` and ``csrc/layer_norm.cu`` (library
``rows``): recurrent mixers with a float32 matrix state per head, short causal convolutions
over time with their kept inputs, norms in groups, the depth-weighted mix of layer outputs, and
gated activations with clamps.

``CudaOps`` inherits these methods; each library is built when one of its kernels is first called, so
a model without a recurrence never compiles ``state``, and one without any of these parts neither.

causal_conv(x, w, step, state, offset, out, add_input, silu)   y = [x +] conv(x) [silu], rows before a portion from the state
conv_tail_store(x, taps, step, state, offset)                  the state's kept inputs renewed after a step
group_norm(x, w, eps, groups, out | residual, rows)            RMS norm in equal consecutive parts of a row
embed_bigram(table, bigram, tokens, ...)                       two tables' rows added, the second's by a hash of two tokens
rmsnorm_shift(x, w, eps, mu, step, state, out, shifted)        RMS norm, and its rows shifted towards the token before
gated_add(y, target)                                           x += scale sigmoid(gate + bias) y
low_rank_decay(low, a2, bias, tau, out)                        sigmoid(low a2^T + bias)^(1/tau)
gated_recurrence(...)                                          a linear recurrence per channel with its gates
tanh_norm(x, alpha, w, b, out | residual, rows)                tanh(alpha x) w + b, the norm without mean or variance
tanh_norm_pair(y, ..., residual, ..., out)                     residual += norm1(y); out = norm2(residual)
layer_norm(x, w, b, eps, out, rows)                            (x - mean) / sqrt(var + eps) w + b
norm_sum(a, b, wa, wb, eps, target, then)                      x += scale (rms(a) wa + rms(b) wb), then a layer norm of x
cap_rows(x, cap)                                               x = cap tanh(x / cap), in place
add_row(x, row)                                                x[t] += row
depth_mix(x, hist, index, weights)                             hist[index] = x; x = sum_j weights[j] hist[j]
add_scaled(dst, a, sa, b, sb)                                  dst += sa a + sb b
glu_rows(gu, interleaved, kind, limit, alpha, out)             out = act(gate, up)
matrix_state(mode, ...)                                        the gated delta rule / the gated sum / the decayed sum of outer products
"""
from __future__ import annotations

import ctypes

import torch

from .build import load_library

_CODE = {torch.float32: 0, torch.bfloat16: 1}
_vp, _i, _f, _ll = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong

GLU_KINDS = {"silu": 0, "clamped": 1, "gelu_tanh": 2}
UNARY_KINDS = {"relu2": 16}              # activations of one value, of feed-forwards without a gate
STATE_MODES = {"delta": 0, "gated_sum": 1, "decayed_sum": 2}
GATE_ACTS = {"silu": 0, "sigmoid": 1}


def _ptr(t):
    return None if t is None else t.data_ptr()


def matrix_state_floats(mode: str, heads: int, dk: int, dv: int) -> int:
    """Floats of state a request keeps for one layer of the recurrence ``mode``."""
    return heads * dk * (dv + 1) + heads if mode == "gated_sum" else heads * dk * dv


class BlockGates:
    """Two block-diagonal matrices ``[blocks, per, per]`` (``[out, in]``) side by side, in the layouts of
    ``gated_recurrence``'s forms: ``rows`` ``[blocks, 2 per, per]`` (the first matrix's rows first), ``cols``
    ``[blocks, per, 2 per]``, and ``thrice`` ``[blocks, 2 per, 3 per]``, ``rows`` three times along ``k`` (made
    when first asked for)."""

    def __init__(self, wr, wi):
        self.blocks, self.per = int(wr.shape[0]), int(wr.shape[1])
        self.rows = torch.cat([wr, wi], dim=1).contiguous()
        self.cols = self.rows.transpose(1, 2).contiguous()
        self._thrice = None
        self._tiles: dict = {}

    @property
    def thrice(self):
        if self._thrice is None:
            self._thrice = self.rows.repeat(1, 1, 3).contiguous()
        return self._thrice

    def tiles(self, per_block: int, device):
        """For a grouped product of ``per_block`` row tiles a block: the block of every tile, and their count."""
        if per_block not in self._tiles:
            self._tiles[per_block] = (
                torch.arange(self.blocks, dtype=torch.int32, device=device).repeat_interleave(per_block),
                torch.full((1,), self.blocks * per_block, dtype=torch.int32, device=device))
        return self._tiles[per_block]


class StateOps:
    _state_lib = None
    cut_state_columns = True          # long portions of few requests: a head's columns over several blocks

    _rows_lib = None
    _channels_lib = None

    @property
    def state_lib(self):
        if self._state_lib is None:
            b = load_library("state")
            b.ti_last_error.restype = ctypes.c_char_p
            b.ti_matrix_state.argtypes = [_i, _vp, _vp, _vp, _i, _i, _i, _vp, _i, _vp, _i, _vp, _i, _vp, _vp, _f, _vp, _i,
                                          _i, _vp, _i, _f, _vp, _vp, _i, _i, _vp, _ll, _i, _i, _i, _i, _i, _vp, _i, _vp,
                                          _vp, _vp]
            self._state_lib = b
        return self._state_lib

    @property
    def channels_lib(self):
        if self._channels_lib is None:
            b = load_library("channels")
            b.ti_last_error.restype = ctypes.c_char_p
            b.ti_low_rank_decay.argtypes = [_vp, _i, _i, _vp, _i, _vp, _f, _i, _i, _vp, _vp]
            b.ti_gated_recurrence.argtypes = [_vp, _i, _vp, _ll, _ll, _vp, _i, _vp, _i, _vp, _vp, _vp, _vp, _i, _i, _vp,
                                              _ll, _vp, _i, _vp]
            b.ti_gated_recurrence_single_supported.argtypes = [_i]
            b.ti_gated_recurrence_single.argtypes = [_vp, _i, _vp, _i, _vp, _i, _vp, _i, _vp, _vp, _vp, _vp, _i, _i, _vp,
                                                     _ll, _vp, _i, _vp]
            b.ti_split_rows.argtypes = [_vp, _i, _i, _i, _i, _i, _vp, _vp]
            self._channels_lib = b
        return self._channels_lib

    @property
    def rows_lib(self):
        if self._rows_lib is None:
            b = load_library("rows")
            b.ti_last_error.restype = ctypes.c_char_p
            b.ti_causal_conv_rows.argtypes = [_vp, _i, _vp, _i, _i, _i, _vp, _vp, _vp, _vp, _ll, _ll, _i, _i, _i, _vp, _vp,
                                              _vp, _i, _i, _vp]
            b.ti_conv_tail_store.argtypes = [_vp, _i, _i, _i, _vp, _vp, _i, _vp, _ll, _ll, _vp, _vp]
            b.ti_embed_bigram.argtypes = [_vp, _vp, _i, _vp, _i, _i, _i, _ll, _ll, _ll, _vp, _vp, _vp, _vp, _vp, _ll, _vp, _vp]
            b.ti_rmsnorm_shift.argtypes = [_vp, _i, _i, _vp, _f, _vp, _vp, _vp, _vp, _vp, _ll, _vp, _vp, _i, _vp]
            b.ti_gated_add.argtypes = [_vp, _i, _vp, _i, _vp, _i, _vp, _f, _i, _i, _vp]
            b.ti_group_norm_rows.argtypes = [_vp, _vp, _vp, _i, _i, _i, _f, _vp, _i, _vp, _i, _vp]
            b.ti_tanh_norm_rows.argtypes = [_vp, _vp, _i, _i, _f, _vp, _vp, _vp, _i, _vp, _i, _vp]
            b.ti_tanh_norm_pair.argtypes = [_vp, _i, _i, _f, _vp, _vp, _vp, _i, _f, _vp, _vp, _vp, _i, _vp]
            b.ti_layer_norm_rows.argtypes = [_vp, _vp, _vp, _vp, _i, _i, _f, _vp, _i, _vp]
            b.ti_norm_sum_rows.argtypes = [_vp, _vp, _vp, _vp, _f, _f, _vp, _i, _i, _i, _vp, _vp, _f, _vp, _i, _vp]
            b.ti_unary_rows.argtypes = [_vp, _ll, _i, _vp, _i, _vp]
            b.ti_cap_rows.argtypes = [_vp, _ll, _f, _vp]
            b.ti_add_row.argtypes = [_vp, _i, _vp, _i, _i, _vp]
            b.ti_depth_mix.argtypes = [_vp, _vp, _ll, _i, _vp, _vp]
            b.ti_add_scaled.argtypes = [_vp, _i, _vp, _f, _vp, _f, _i, _i, _vp]
            b.ti_glu_rows.argtypes = [_vp, _i, _i, _i, _i, _f, _f, _vp, _i, _vp]
            self._rows_lib = b
        return self._rows_lib

    def _rw(self, rc: int) -> None:
        self._ok(rc, self.rows_lib)

    def _ch(self, rc: int) -> None:
        self._ok(rc, self.channels_lib)

    def _st(self, rc: int) -> None:
        self._ok(rc, self.state_lib)

    @staticmethod
    def _want(cond: bool, msg: str) -> None:
        if not cond:
            from .cuda_ops import KernelError
            raise KernelError(msg)

    # ---- short convolutions over time ----------------------------------------------------------
    def causal_conv(self, x, w, step, state, state_offset, out, add_input=False, silu=False, renew=False, in_bias=None,
                    bias=None):
        """``out[t, c] = [x[t, c] +] sum_j w[c, j] x[t - taps + 1 + j, c]``, then silu if asked, over
        float32 rows ``x`` (a column slice is fine).  Rows before a request's portion come from
        ``state`` (a ``StateView``: per slot ``[taps - 1, channels]`` floats from ``state_offset``
        on, the newest row last).  ``w`` None: the rows are converted (and nothing else).
        ``in_bias`` (float32 per channel) is added to every row of ``x`` before anything else (the kept
        rows hold it already), ``bias`` to the convolution's result.  ``renew``: the kept rows become the requests' last inputs after this step, in the same
        launch where every request brings one token, else by ``conv_tail_store`` behind it."""
        t, c = x.shape
        taps = 0 if w is None else w.shape[1]
        self._want(x.dtype == torch.float32 and x.stride(1) == 1 and out.stride(1) == 1
                   and tuple(out.shape) == (t, c), "causal_conv: float32 rows in, rows of the same shape out")
        self._want(w is None or (w.dtype == torch.float32 and w.is_contiguous() and w.shape[0] == c),
                   "causal_conv: float32 weights [channels, taps]")
        st = None if state is None else state.state
        self._want(taps <= 1 or (st is not None and st.dtype == torch.float32
                                 and st[0].numel() >= state_offset + (taps - 1) * c),
                   "causal_conv: the state must hold taps - 1 float32 rows")
        renew = bool(renew) and taps > 1 and state.writes
        in_place = renew and step.max_q_len == 1 and step.num_requests == t
        self._rw(self.rows_lib.ti_causal_conv_rows(
            x.data_ptr(), x.stride(0), _ptr(w), taps, c, t, step.req_of_tok.data_ptr(), step.cu_q.data_ptr(),
            _ptr(state.slots) if state is not None else None, _ptr(st), st.stride(0) if st is not None else 0,
            int(state_offset), int(bool(add_input)), int(bool(silu)), int(in_place), _ptr(in_bias), _ptr(bias),
            out.data_ptr(), _CODE[out.dtype], out.stride(0), self._stream()))
        if renew and not in_place:
            self.conv_tail_store(x, taps, step, state, state_offset, in_bias)

    def conv_tail_store(self, x, taps, step, state, state_offset, in_bias=None):
        """The state's ``taps - 1`` kept rows of every request become its last inputs after this
        step.  Launched behind every reader of the old rows."""
        if taps <= 1 or not state.writes:
            return
        c = x.shape[1]
        st = state.state
        self._want(x.dtype == torch.float32 and x.stride(1) == 1, "conv_tail_store: float32 rows")
        self._rw(self.rows_lib.ti_conv_tail_store(
            x.data_ptr(), x.stride(0), int(taps), c, step.cu_q.data_ptr(), state.slots.data_ptr(),
            step.num_requests, st.data_ptr(), st.stride(0), int(state_offset), _ptr(in_bias), self._stream()))

    # ---- what the last token of a request leaves behind -------------------------------------------
    def embed_bigram(self, table, bigram, token_ids, buckets, mul_prev, mul_cur, step, state, out):
        """``out[t] = table[token[t]] + bigram[row]`` in float32, ``row = (token before * mul_prev +
        token[t] * mul_cur) mod buckets``, or ``buckets`` for a request's first token (position 0).  The
        token before a portion is the int32 that ``state`` keeps, which then becomes the portion's last."""
        t, n = out.shape
        st = state.state
        self._want(out.dtype == torch.float32 and out.is_contiguous() and token_ids.dtype == torch.int32
                   and token_ids.shape[0] == t and table.dtype == bigram.dtype and table.is_contiguous()
                   and bigram.is_contiguous() and table.shape[1] == bigram.shape[1] == n
                   and bigram.shape[0] == buckets + 1, "embed_bigram: two tables of one dtype and width, float32 rows out")
        self._want(st is not None and st.dtype == torch.int32 and state.writes, "embed_bigram: the state keeps an int32")
        self._rw(self.rows_lib.ti_embed_bigram(
            table.data_ptr(), bigram.data_ptr(), _CODE[table.dtype], token_ids.data_ptr(), t, n, table.shape[0],
            int(buckets), int(mul_prev), int(mul_cur), step.positions.data_ptr(), step.req_of_tok.data_ptr(),
            step.cu_q.data_ptr(), state.slots.data_ptr(), st.data_ptr(), st.stride(0), out.data_ptr(), self._stream()))

    def rmsnorm_shift(self, x, weight, eps, mu, step, state, out, shifted):
        """``out = h`` and ``shifted = h + (h' - h) mu`` with ``h`` the RMS-normed rows of ``x`` and ``h'``
        the row of the token before: the row above, or for a portion's first token the float32 row
        that ``state`` keeps, which then becomes the portion's last ``h``."""
        self.flush()
        t, n = x.shape
        st = state.state
        self._want(x.dtype == torch.float32 and x.is_contiguous() and out.dtype == shifted.dtype and out.is_contiguous()
                   and shifted.is_contiguous() and tuple(out.shape) == tuple(shifted.shape) == (t, n),
                   "rmsnorm_shift: float32 rows in, two outputs of their shape")
        for v in (weight, mu):
            self._want(v.dtype == torch.float32 and v.is_contiguous() and v.shape[0] == n,
                       "rmsnorm_shift: float32 weight and shift per element")
        self._want(st is not None and st.dtype == torch.float32 and st[0].numel() >= n and state.writes,
                   "rmsnorm_shift: the state keeps one float32 row")
        self._rw(self.rows_lib.ti_rmsnorm_shift(
            x.data_ptr(), t, n, weight.data_ptr(), float(eps), mu.data_ptr(), step.req_of_tok.data_ptr(),
            step.cu_q.data_ptr(), state.slots.data_ptr(), st.data_ptr(), st.stride(0), out.data_ptr(), shifted.data_ptr(),
            _CODE[out.dtype], self._stream()))

    # ---- sums that pass a gate ---------------------------------------------------------------------
    def gated_add(self, y, target):
        """``x += scale * sigmoid(gate + bias) * y`` (or, without a gate, ``x += scale * y``) for a
        ``parts.base.GatedSum`` ``target``."""
        self.flush()
        x, gate, bias = target.x, target.gate, target.bias
        if gate is None:
            self.add_scaled(x, y, target.scale)
            return
        for v in (x, gate, y):
            self._want(v.dtype == torch.float32 and v.stride(1) == 1 and tuple(v.shape) == tuple(x.shape),
                       "gated_add: float32 rows of one shape")
        self._want(bias.dtype == torch.float32 and bias.is_contiguous() and bias.shape[0] == x.shape[1],
                   "gated_add: a float32 bias per element")
        self._rw(self.rows_lib.ti_gated_add(x.data_ptr(), x.stride(0), y.data_ptr(), y.stride(0), gate.data_ptr(),
                                            gate.stride(0), bias.data_ptr(), float(target.scale), x.shape[0], x.shape[1],
                                            self._stream()))

    # ---- norms in groups, depth mix, sums ---------------------------------------------------------
    def group_norm(self, x, weight, eps, groups, out=None, rows=None, residual=None):
        """RMS norm of every row of ``x`` in ``groups`` equal consecutive parts (each divided by its
        own ``sqrt(mean(part^2) + eps)``), times ``weight``: stored in ``out`` (of the rows ``rows``
        if given), or added to the float32 ``residual``."""
        n = x.shape[1]
        self._want(x.dtype == torch.float32 and x.is_contiguous() and weight.dtype == torch.float32
                   and weight.shape[0] == n, "group_norm: float32 rows and a float32 weight per element")
        self._want(n % groups == 0, f"group_norm: {n} elements do not fall into {groups} equal groups")
        num = x.shape[0] if rows is None else rows.shape[0]
        if residual is not None:
            self._want(rows is None and residual.dtype == torch.float32 and residual.stride(1) == 1
                       and tuple(residual.shape) == tuple(x.shape), "group_norm: a float32 residual of x's shape")
        else:
            self._want(out is not None and out.is_contiguous() and tuple(out.shape) == (num, n), "group_norm: out")
        self._rw(self.rows_lib.ti_group_norm_rows(
            x.data_ptr(), weight.data_ptr(), _ptr(rows), num, n, int(groups), float(eps), _ptr(out),
            _CODE[out.dtype] if out is not None else 0, _ptr(residual),
            residual.stride(0) if residual is not None else 0, self._stream()))

    def tanh_norm(self, x, alpha, weight, bias, out=None, rows=None, residual=None):
        """``tanh(alpha x) weight + bias`` for every row of the float32 ``x`` (one scalar ``alpha``, a
        weight and, if not None, a bias per element): stored in ``out`` (of the rows ``rows`` if given),
        or added to the float32 ``residual``."""
        n = x.shape[1]
        self._want(x.dtype == torch.float32 and x.is_contiguous() and weight.dtype == torch.float32
                   and weight.is_contiguous() and weight.shape[0] == n
                   and (bias is None or (bias.dtype == torch.float32 and bias.is_contiguous() and bias.shape[0] == n)),
                   "tanh_norm: float32 rows, a float32 weight and bias per element")
        num = x.shape[0] if rows is None else rows.shape[0]
        if residual is not None:
            self._want(rows is None and residual.dtype == torch.float32 and residual.stride(1) == 1
                       and tuple(residual.shape) == tuple(x.shape), "tanh_norm: a float32 residual of x's shape")
        else:
            self._want(out is not None and out.is_contiguous() and tuple(out.shape) == (num, n)
                       and (rows is None or rows.dtype == torch.int32), "tanh_norm: out")
        self._rw(self.rows_lib.ti_tanh_norm_rows(
            x.data_ptr(), _ptr(rows), num, n, float(alpha), weight.data_ptr(), _ptr(bias), _ptr(out),
            _CODE[out.dtype] if out is not None else 0, _ptr(residual),
            residual.stride(0) if residual is not None else 0, self._stream()))

    def tanh_norm_pair(self, y, alpha1, weight1, bias1, residual, alpha2, weight2, bias2, out):
        """``residual += tanh(alpha1 y) weight1 + bias1``, then ``out = tanh(alpha2 residual) weight2 +
        bias2``: the norm behind one sublayer and the norm in front of the next, in one launch.  The
        float32 sum is the same as by ``tanh_norm`` twice."""
        n = y.shape[1]
        self._want(y.dtype == torch.float32 and y.is_contiguous() and residual.dtype == torch.float32
                   and residual.stride(1) == 1 and tuple(residual.shape) == tuple(y.shape) and out.is_contiguous()
                   and tuple(out.shape) == tuple(y.shape), "tanh_norm_pair: float32 rows, a residual and an output of their shape")
        for v in (weight1, bias1, weight2, bias2):
            self._want(v is None or (v.dtype == torch.float32 and v.is_contiguous() and v.shape[0] == n),
                       "tanh_norm_pair: float32 weights and biases per element")
        self._rw(self.rows_lib.ti_tanh_norm_pair(
            y.data_ptr(), y.shape[0], n, float(alpha1), weight1.data_ptr(), _ptr(bias1), residual.data_ptr(),
            residual.stride(0), float(alpha2), weight2.data_ptr(), _ptr(bias2), out.data_ptr(), _CODE[out.dtype],
            self._stream()))

    def layer_norm(self, x, weight, bias, eps, out, rows=None):
        """``(x - mean) / sqrt(var + eps) * weight + bias`` for every row of the float32 ``x`` (of the rows ``rows`` if
        given), ``var`` the mean of the squared deviations."""
        n = x.shape[1]
        num = x.shape[0] if rows is None else rows.shape[0]
        self._want(x.dtype == torch.float32 and x.is_contiguous() and out.is_contiguous() and tuple(out.shape) == (num, n)
                   and (rows is None or rows.dtype == torch.int32), "layer_norm: contiguous float32 rows, rows of the same length out")
        for v in (weight, bias):
            self._want(v.dtype == torch.float32 and v.is_contiguous() and v.shape[0] == n,
                       "layer_norm: a float32 weight and bias per element")
        self._rw(self.rows_lib.ti_layer_norm_rows(x.data_ptr(), weight.data_ptr(), bias.data_ptr(), _ptr(rows), num, n,
                                                  float(eps), out.data_ptr(), _CODE[out.dtype], self._stream()))

    def norm_sum(self, a, b, weight_a, weight_b, eps, residual, scale, then=None):
        """``residual += scale * (rms(a) * weight_a + rms(b) * weight_b)``, every row of ``a`` and ``b`` over the root of its
        mean square (+ ``eps``).  ``then = (weight, bias, eps, out)``: ``out`` gets the layer norm of the new rows in the
        same launch."""
        t, n = a.shape
        for v in (a, b):
            self._want(v.dtype == torch.float32 and v.is_contiguous() and tuple(v.shape) == (t, n), "norm_sum: float32 rows of one shape")
        for v in (weight_a, weight_b, *(then[:2] if then is not None else ())):
            self._want(v.dtype == torch.float32 and v.is_contiguous() and v.shape[0] == n, "norm_sum: a float32 weight per element")
        self._want(residual.dtype == torch.float32 and residual.stride(1) == 1 and tuple(residual.shape) == (t, n),
                   "norm_sum: a float32 residual of the rows' shape")
        w2, b2, eps2, out = then if then is not None else (None, None, 0.0, None)
        self._want(out is None or (out.is_contiguous() and tuple(out.shape) == (t, n)), "norm_sum: the normed rows out")
        self._rw(self.rows_lib.ti_norm_sum_rows(
            a.data_ptr(), b.data_ptr(), weight_a.data_ptr(), weight_b.data_ptr(), float(eps), float(scale),
            residual.data_ptr(), residual.stride(0), t, n, _ptr(w2), _ptr(b2), float(eps2), _ptr(out),
            _CODE[out.dtype] if out is not None else 0, self._stream()))

    def unary_rows(self, x, kind, out):
        """``out = act(x)`` element by element over a contiguous float32 tensor; ``kind`` "relu2": the square of relu."""
        self._want(x.dtype == torch.float32 and x.is_contiguous() and out.is_contiguous() and out.shape == x.shape,
                   "unary_rows: contiguous float32 in, the same shape out")
        self._rw(self.rows_lib.ti_unary_rows(x.data_ptr(), x.numel(), UNARY_KINDS[kind], out.data_ptr(), _CODE[out.dtype],
                                             self._stream()))

    def cap_rows(self, x, cap):
        """``x = cap tanh(x / cap)`` over a contiguous float32 tensor, in place."""
        self._want(x.dtype == torch.float32 and x.is_contiguous(), "cap_rows: contiguous float32")
        self._rw(self.rows_lib.ti_cap_rows(x.data_ptr(), x.numel(), float(cap), self._stream()))

    def add_row(self, x, row):
        """``x[t] += row`` for every row of the float32 ``x``."""
        self._want(x.dtype == torch.float32 and x.stride(1) == 1 and row.dtype == torch.float32 and row.is_contiguous()
                   and row.numel() == x.shape[1], "add_row: float32 rows and one float32 row of their length")
        self._rw(self.rows_lib.ti_add_row(x.data_ptr(), x.stride(0), row.data_ptr(), x.shape[0], x.shape[1],
                                           self._stream()))

    def depth_mix(self, x, hist, index, weights=None):
        """``hist[index] = x`` and, with ``weights`` (float32, ``index + 1`` of them),
        ``x = sum_{j <= index} weights[j] hist[j]``; ``x`` float32 ``[T, width]``, ``hist``
        ``[n, T, width]``."""
        self._want(x.dtype == torch.float32 and x.is_contiguous() and hist.dtype == torch.float32
                   and hist.is_contiguous() and tuple(hist.shape[1:]) == tuple(x.shape) and 0 <= index < hist.shape[0],
                   "depth_mix: float32 rows and a history of such rows")
        self._want(weights is None or (weights.dtype == torch.float32 and weights.is_contiguous()
                                       and weights.shape[0] == index + 1), "depth_mix: index + 1 float32 weights")
        self._rw(self.rows_lib.ti_depth_mix(x.data_ptr(), hist.data_ptr(), x.numel(), int(index), _ptr(weights),
                                             self._stream()))

    def add_scaled(self, dst, a, sa, b=None, sb=0.0):
        """``dst += sa * a [+ sb * b]`` over float32 rows."""
        self._want(dst.dtype == torch.float32 and dst.stride(1) == 1 and a.dtype == torch.float32 and a.is_contiguous()
                   and tuple(a.shape) == tuple(dst.shape)
                   and (b is None or (b.dtype == torch.float32 and b.is_contiguous() and b.shape == a.shape)),
                   "add_scaled: float32 rows of one shape")
        self._rw(self.rows_lib.ti_add_scaled(dst.data_ptr(), dst.stride(0), a.data_ptr(), float(sa), _ptr(b), float(sb),
                                              dst.shape[0], dst.shape[1], self._stream()))

    def glu_rows(self, gu, interleaved, kind, limit, alpha, out):
        """``out = act(gate, up)`` over the float32 product ``gu`` ``[T, 2 n]`` that holds gate and up
        columns stacked or, ``interleaved``, in strips of 8 and 8.  ``kind`` "silu": ``silu(g) u``;
        "clamped": ``g = min(g, limit)``, ``u = clamp(u, -limit, limit)``, ``g sigmoid(alpha g) (u + 1)``;
        "gelu_tanh": ``gelu(g) u`` (the tanh form)."""
        t, n = out.shape
        self._want(gu.dtype == torch.float32 and gu.is_contiguous() and tuple(gu.shape) == (t, 2 * n)
                   and out.is_contiguous(), "glu_rows: a float32 product of gate and up columns")
        self._rw(self.rows_lib.ti_glu_rows(gu.data_ptr(), t, n, int(bool(interleaved)), GLU_KINDS[kind], float(limit),
                                            float(alpha), out.data_ptr(), _CODE[out.dtype], self._stream()))

    # ---- recurrences per channel -----------------------------------------------------------------------
    def low_rank_decay(self, low, a2, bias, tau, out):
        """``out = sigmoid(low a2^T + bias)^(1 / tau)`` in float32; ``low`` float32 ``[T, rank]`` (a column
        slice is fine), ``a2`` ``[n, rank]``, ``bias`` float32 ``[n]``."""
        t, n = out.shape
        self._want(low.dtype == torch.float32 and low.stride(1) == 1 and low.shape[0] == t and out.dtype == torch.float32
                   and out.is_contiguous() and a2.is_contiguous() and tuple(a2.shape) == (n, low.shape[1])
                   and bias.dtype == torch.float32 and bias.is_contiguous() and bias.shape[0] == n and float(tau) > 0.0,
                   "low_rank_decay: float32 rows, a matrix [n, rank] and a float32 bias per column")
        self._ch(self.channels_lib.ti_low_rank_decay(
            low.data_ptr(), low.stride(0), low.shape[1], a2.data_ptr(), _CODE[a2.dtype], bias.data_ptr(), 1.0 / float(tau),
            t, n, out.data_ptr(), self._stream()))

    def pack_block_gates(self, wr, wi):
        """The two block-diagonal matrices ``[blocks, per, per]`` of ``gated_recurrence`` in the layouts
        that its forms read."""
        return BlockGates(wr, wi)

    def gated_recurrence(self, u, gates, gate_bias, log_decay, y, y_bias, step, state, out):
        """One linear recurrence per channel with block-diagonal gates, all tokens of the step in order,
        from and into each request's state (``state``: one float32 per channel at the start of its slot):

            zr, zi = Wr[b] u_b, Wi[b] u_b                     (``gates`` from ``pack_block_gates``)
            a = exp(log_decay * sigmoid(zr + br));   S <- a S + sqrt(1 - a^2) sigmoid(zi + bi) u
            out = S * gelu(y + y_bias)

        ``u``, ``y`` float32 ``[T, width]`` (column slices are fine); ``gate_bias`` ``[2, width]`` (``br``,
        ``bi``), ``log_decay`` (at most 0) and ``y_bias`` ``[width]``.  The products have float32 sums of
        the float32 ``u``: on CUDA cores, or, for the many rows of a bfloat16 step, as a grouped
        tensor-core product over ``u`` cut into three bfloat16 parts."""
        t, n = out.shape
        st = state.state
        for name, x in (("u", u), ("y", y)):
            self._want(x.dtype == torch.float32 and x.stride(1) == 1 and tuple(x.shape) == (t, n),
                       f"gated_recurrence: {name} must be float32 [T, {n}]")
        for x, count in ((gate_bias, 2 * n), (log_decay, n), (y_bias, n)):
            self._want(x.dtype == torch.float32 and x.is_contiguous() and x.numel() == count,
                       "gated_recurrence: float32 vectors per channel")
        self._want(st is not None and st.dtype == torch.float32 and st[0].numel() >= n and st.stride(-1) == 1
                   and state.writes, "gated_recurrence: the state holds one float32 per channel")
        blocks, per = gates.blocks, gates.per
        self._want(blocks * per == n and out.is_contiguous(), "gated_recurrence: equal blocks, contiguous rows out")
        lib = self.channels_lib
        # a row's bits of a float32 step must not depend on the step around it: one form for all of them
        fast = out.dtype == torch.bfloat16
        if (fast and step.max_q_len == 1 and step.num_requests == t and gates.rows.data_ptr() % 16 == 0
                and lib.ti_gated_recurrence_single_supported(per)):
            self._ch(lib.ti_gated_recurrence_single(
                u.data_ptr(), u.stride(0), gates.rows.data_ptr(), _CODE[gates.rows.dtype], y.data_ptr(), y.stride(0),
                gate_bias.data_ptr(), per, log_decay.data_ptr(), y_bias.data_ptr(), step.cu_q.data_ptr(),
                state.slots.data_ptr(), step.num_requests, n, st.data_ptr(), st.stride(0), out.data_ptr(),
                _CODE[out.dtype], self._stream()))
            return
        z, row_stride, block_stride = self.block_products(u, gates, fast)
        self.recurrence_rows(u, z, row_stride, block_stride, gate_bias, per, log_decay, y, y_bias, step, state, out)

    def block_products(self, u, gates, fast):
        """``Wr[b] u_b`` and ``Wi[b] u_b`` for every row of the float32 ``u``, with float32 sums.  Returns the
        float32 rows, the stride from a token to the next and the stride from a block to the next; a
        block's ``per`` columns of the first product lie in front of those of the second.  ``fast``: many
        rows may take the tensor cores."""
        t, n = u.shape
        blocks, per = gates.blocks, gates.per
        if fast and t > 64 and per % 8 == 0 and gates.rows.dtype == torch.bfloat16:
            lib = self.channels_lib
            padded = -(-t // 128) * 128
            cut = torch.empty((blocks, padded, 3 * per), dtype=torch.bfloat16, device=u.device)
            self._ch(lib.ti_split_rows(u.data_ptr(), u.stride(0), t, n, per, padded, cut.data_ptr(), self._stream()))
            z = torch.empty((blocks, padded, 2 * per), dtype=torch.float32, device=u.device)
            group_of_tile, tiles = gates.tiles(padded // 128, u.device)
            self._ok(self.bf16.ti_gemm_tcgen05_grouped(
                cut.data_ptr(), gates.thrice.data_ptr(), z.data_ptr(), None, blocks * padded, 2 * per, 3 * per, 3 * per,
                3 * per, 2 * per, 0, 0, blocks, group_of_tile.data_ptr(), tiles.data_ptr(), self.status.data_ptr(),
                self._stream()), self.bf16)
            return z, 2 * per, padded * 2 * per
        z = torch.empty((t, blocks, 2 * per), dtype=torch.float32, device=u.device)
        if per <= 768:
            self.head_project(u.unflatten(1, (blocks, per)), gates.cols, z)
        else:
            for b in range(blocks):
                self.linear(u[:, b * per:(b + 1) * per], gates.rows[b], z[:, b])
        return z, 2 * n, 2 * per

    def recurrence_rows(self, u, z, row_stride, block_stride, gate_bias, per, log_decay, y, y_bias, step, state, out):
        """The walk of ``gated_recurrence`` behind its products (``z`` and its strides: ``block_products``)."""
        t, n = out.shape
        st = state.state
        self._ch(self.channels_lib.ti_gated_recurrence(
            u.data_ptr(), u.stride(0), z.data_ptr(), row_stride, block_stride, y.data_ptr(), y.stride(0),
            gate_bias.data_ptr(), per, log_decay.data_ptr(), y_bias.data_ptr(), step.cu_q.data_ptr(),
            state.slots.data_ptr(), step.num_requests, n, st.data_ptr(), st.stride(0), out.data_ptr(), _CODE[out.dtype],
            self._stream()))

    # ---- recurrences over a matrix state -------------------------------------------------------------
    def matrix_state(self, mode, q, k, v, s0, s1, c0, c1, step, state, out, *, heads, kv_heads, dk, dv, eps,
                     norm_weight, norm_per_row=False, gate=None, gate_act="silu", cap=0.0, decay=None):
        """One step of a recurrent mixer with a float32 matrix state ``[dk, dv]`` per head, for all
        tokens of the step in order, from and into each request's state slot (``state``: a
        ``StateView`` of ``matrix_state_floats`` floats).

        ``mode`` "delta" (the gated delta rule): ``q, k`` float32 rows of ``kv_heads x dk`` (brought to
        unit length here, q also times ``dk^-1/2``), ``v`` of ``heads x dv``; ``s0`` the logit of beta and
        ``s1`` the decay's argument per (token, head); ``c0 = A_log``, ``c1 = dt_bias`` per head.
        ``mode`` "gated_sum" (exponential gates under a running maximum): ``s0, s1`` the input and forget
        gates' pre-activations, ``c0, c1`` their biases, ``cap`` the bound of ``cap tanh(. / cap)``.
        ``mode`` "decayed_sum": ``decay`` float32 rows like ``k``, the factor of every row of ``S``; ``q``
        times ``dk^-1/2``; no per-head scalars.

        Each head's output is brought to unit root mean square over ``dv`` (``eps``), multiplied by
        ``norm_weight`` (``[dv]``, or ``[heads * dv]`` with ``norm_per_row``) and by ``act(gate)``
        (float32 ``[T, heads * dv]``; "silu" or "sigmoid"), and written to ``out`` ``[T, heads * dv]``."""
        t = q.shape[0]
        st = state.state
        need = matrix_state_floats(mode, heads, dk, dv)
        rows = [("q", q, kv_heads * dk), ("k", k, kv_heads * dk), ("v", v, heads * dv)]
        decayed = mode == "decayed_sum"
        rows += [("decay", decay, kv_heads * dk)] if decayed else [("s0", s0, heads), ("s1", s1, heads)]
        for name, x, width in rows:
            self._want(x.dtype == torch.float32 and x.stride(1) == 1 and x.shape[0] == t and x.shape[1] == width,
                       f"matrix_state: {name} must be float32 [T, {width}]")
        for name, x in () if decayed else (("c0", c0), ("c1", c1)):
            self._want(x.dtype == torch.float32 and x.is_contiguous() and x.shape[0] == heads,
                       f"matrix_state: {name} must hold one float32 per head")
        self._want(norm_weight.dtype == torch.float32 and norm_weight.is_contiguous()
                   and norm_weight.shape[0] == (heads * dv if norm_per_row else dv), "matrix_state: the norm's weight")
        self._want(gate is None or (gate.dtype == torch.float32 and gate.stride(1) == 1 and gate.shape[0] == t
                                    and gate.shape[1] == heads * dv), "matrix_state: the gate must be float32 [T, heads * dv]")
        self._want(st is not None and st.dtype == torch.float32 and st[0].numel() >= need and st.stride(-1) == 1,
                   f"matrix_state: the state must hold {need} float32 values per request")
        self._want(out.is_contiguous() and tuple(out.shape) == (t, heads * dv), "matrix_state: out")
        self._want(state.writes, "matrix_state: a recurrence renews its state")
        # few (request, head) pairs with long portions: a head's columns over several blocks
        col_block, o_raw, carry = 0, None, None
        pairs = step.num_requests * heads
        if dv > 128 or (self.cut_state_columns and dv >= 16 and step.max_q_len > 64 and pairs <= 2 * self.num_sms):
            col_block = 16 if decayed and dk > 64 else 8      # over wide keys a thread walks two columns
            while col_block < 128 and pairs * -(-dv // col_block) > 4 * self.num_sms:
                col_block *= 2
            o_raw = torch.empty((t, heads * dv), dtype=torch.float32, device=q.device)
            self.launches += 1
            if mode == "gated_sum":
                carry = torch.empty((pairs, dk + 1), dtype=torch.float32, device=q.device)
                self.launches += 1
        self._st(self.state_lib.ti_matrix_state(
            STATE_MODES[mode], q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), k.stride(0), v.stride(0),
            _ptr(s0), 0 if decayed else s0.stride(0), _ptr(s1), 0 if decayed else s1.stride(0), _ptr(decay),
            decay.stride(0) if decayed else 0, _ptr(c0), _ptr(c1), float(cap),
            _ptr(gate), gate.stride(0) if gate is not None else 0, GATE_ACTS[gate_act], norm_weight.data_ptr(),
            int(bool(norm_per_row)), float(eps), step.cu_q.data_ptr(), state.slots.data_ptr(), step.num_requests, t,
            st.data_ptr(), st.stride(0), heads, kv_heads, dk, dv, col_block, out.data_ptr(), _CODE[out.dtype],
            _ptr(o_raw), _ptr(carry), self._stream()))
