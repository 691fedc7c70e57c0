"""Recurrences whose state decays by one number per head, behind a short causal convolution, and the operators around them.

    short_conv        act(causal convolution over time, per channel); a sequence's last inputs are part of its state
    head_recurrence   gated delta rule, or state-space form with a scalar decay, over the new tokens of every sequence
    gated_group_norm  norm_w * RMS norm (in equal parts of the row) of y * act(gate)

CUDA tensors run csrc/kernels/head_recurrence.cu; CPU tensors run the PyTorch statement of the same op.
"""

from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Tuple

import torch
import torch.nn.functional as F

from . import _lib
from . import _count_launch, _native, _ptr, _stream
from .linear_attention import linear_state_shape
from .mixers import ACTIVATIONS, Proj, _ref, gate_heads

UNIT_EPS = 1e-6


@dataclass
class ShortConv:
    """Weights w fp32 [taps, channels] (the last row for the current token), bias fp32 [channels] or None."""
    w: torch.Tensor
    bias: Optional[torch.Tensor] = None

    @property
    def taps(self) -> int:
        return self.w.shape[0]

    @property
    def state_shape(self) -> Tuple[int, int]:
        """Inputs of a sequence's last tokens: that of position p in row p % taps."""
        return tuple(self.w.shape)


@dataclass
class HeadRecurrence:
    """Sizes and constants.  Query / key head of head h: h // (heads / groups).  q_col, k_col, v_col: first columns of queries
    [groups * dim], keys [groups * dim] and values [heads * vdim] among the convolved channels.  Decay exp(-rate * dt) with
    dt = softplus(a + dt_bias) (fp32 [heads] each).

    delta: S <- g S; u = sigmoid(b) (v - S^T k); S <- S + k u^T; o = S^T q with unit-length k and q, q times q_scale.
    Otherwise S <- g S + k (dt v)^T; o = q_scale S^T q + skip v."""
    heads: int
    groups: int
    dim: int
    vdim: int
    q_col: int
    k_col: int
    v_col: int
    rate: torch.Tensor
    dt_bias: torch.Tensor
    delta: bool
    q_scale: float = 1.0
    skip: Optional[torch.Tensor] = None
    eps: float = 1e-6

    @property
    def state_shape(self) -> Tuple[int, int, int]:
        return linear_state_shape(self.heads, self.dim, self.vdim)


def _spans(context_lens, q_start, q_lens, rows):
    """(first row, new tokens, context length, slot) of every active sequence, on the host."""
    for b in range(context_lens.shape[0]):
        n = 1 if q_lens is None else int(q_lens[b])
        ctx = int(context_lens[b])
        if n > 0 and ctx >= n:
            yield b if q_start is None else int(q_start[b]), n, ctx, b if rows is None else int(rows[b])


def _conv_ref(x, conv, state, spans, act):
    """x fp32 [T, C]; reads and updates the state."""
    out = torch.zeros_like(x)
    R = conv.taps
    for t0, n, ctx, slot in spans:
        past = [state[slot, p % R] if p >= 0 else torch.zeros_like(x[0]) for p in range(ctx - n - R + 1, ctx - n)]
        full = torch.cat([torch.stack(past), x[t0:t0 + n]]) if past else x[t0:t0 + n]
        y = sum(conv.w[j] * full[j:j + n] for j in range(R))
        out[t0:t0 + n] = y if conv.bias is None else y + conv.bias
        for p in range(max(ctx - n, ctx - R), ctx):
            state[slot, p % R] = x[t0 + p - (ctx - n)]
    return ACTIVATIONS[act][1](out)


def _check_conv(conv: ShortConv, state: torch.Tensor) -> None:
    for t in (conv.w, conv.bias, state):
        if t is not None and (t.dtype != torch.float32 or not t.is_contiguous()):
            raise TypeError("a short convolution wants contiguous fp32 weights and state")
    if tuple(state.shape[1:]) != conv.state_shape:
        raise ValueError(f"state of the convolution must be [slots, {conv.state_shape}]")


def short_conv(x: Proj, conv: ShortConv, state: torch.Tensor, context_lens: torch.Tensor, q_start: torch.Tensor,
               q_lens: torch.Tensor, rows: Optional[torch.Tensor] = None, act: str = "silu",
               dtype: torch.dtype = torch.bfloat16) -> torch.Tensor:
    """``act(sum_j w[j] * x[t - (taps - 1) + j] + bias)`` over the new tokens of every sequence -> [T, channels]; zeros before a
    sequence's first token.  state fp32 [slots, taps, channels] is read and written in place at slot rows[b] (rows None: b);
    context_lens counts the new tokens."""
    T, C = x.t.shape[-2], x.width
    out = torch.empty((T, C), dtype=dtype, device=x.t.device)
    if not _native(out):
        return out.copy_(_conv_ref(x.value(), conv, state, _spans(context_lens, q_start, q_lens, rows), act).to(dtype))
    _check_conv(conv, state)
    rc = _lib.lib().nkb_short_conv(_ref(x), conv.w.data_ptr(), _ptr(conv.bias), state.data_ptr(), _ptr(rows), q_start.data_ptr(),
                                   q_lens.data_ptr(), context_lens.data_ptr(), out.data_ptr(), 1 if dtype == torch.bfloat16 else 0,
                                   context_lens.shape[0], T, C, conv.taps, ACTIVATIONS[act][0], _stream())
    _lib.check(rc, "nkb_short_conv")
    _count_launch(2)
    return out


def _recur_ref(r: HeadRecurrence, y, a, b, state, spans):
    """y fp32 [T, channels] after the convolution -> fp32 [T, heads, vdim]; reads and updates the state."""
    T, per = y.shape[0], r.heads // r.groups
    cut = lambda col, n, d: y[:, col:col + n * d].reshape(T, n, d)
    q, k, v = cut(r.q_col, r.groups, r.dim), cut(r.k_col, r.groups, r.dim), cut(r.v_col, r.heads, r.vdim)
    if r.delta:
        q, k = (x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + UNIT_EPS) for x in (q, k))
    q, k = (x.repeat_interleave(per, 1) for x in (q * r.q_scale, k))
    dt = F.softplus(a + r.dt_bias, threshold=100.0)
    g = torch.exp(-r.rate * dt)
    out = torch.zeros((T, r.heads, r.vdim))
    for t0, n, ctx, slot in spans:
        S = torch.zeros((r.heads, r.vdim, r.dim)) if ctx == n else state[slot, :, :, :r.dim].clone()
        for t in range(t0, t0 + n):
            S = g[t][:, None, None] * S
            if r.delta:
                u = torch.sigmoid(b[t])[:, None] * (v[t] - torch.einsum("hvd,hd->hv", S, k[t]))
            else:
                u = dt[t][:, None] * v[t]
            S = S + u[:, :, None] * k[t][:, None, :]
            out[t] = torch.einsum("hvd,hd->hv", S, q[t])
        state[slot, :, :, :r.dim] = S
    if r.skip is not None:
        out = out + r.skip[:, None] * v
    return out


def head_recurrence(r: HeadRecurrence, x: Proj, conv: ShortConv, a: Proj, b: Optional[Proj], gate: Proj, norm_w: torch.Tensor,
                    state: torch.Tensor, conv_state: torch.Tensor, context_lens: torch.Tensor, *, parts: int = 0,
                    gate_act: str = "silu", q_start: Optional[torch.Tensor] = None, q_lens: Optional[torch.Tensor] = None,
                    rows: Optional[torch.Tensor] = None, dtype: torch.dtype = torch.bfloat16) -> torch.Tensor:
    """The convolution of the channels x, the recurrence over them with decay logits a [T, heads] and write strengths b
    [T, heads] (delta rule only), and the norm and gate of its results o [T, heads * vdim], returned in `dtype`:

        parts 0:   gate_act(gate) * norm_w * o / sqrt(mean(o^2) + eps)   per head, norm_w [vdim]
        otherwise: norm_w * z / sqrt(mean(z^2) + eps) in `parts` equal parts of a row, z = o * gate_act(gate)

    state [slots, heads, vdim, dim_p] and conv_state [slots, taps, channels], fp32, are read and written in place at slot
    rows[b] (rows None: b).  context_lens counts the new tokens; a sequence whose tokens are all new starts from zero, one with
    a negative length is skipped.  q_lens None: one new token per sequence (a decode step)."""
    T, inner = x.t.shape[-2], r.heads * r.vdim
    if r.delta != (b is not None):
        raise ValueError("the delta rule has write strengths, the state-space form has none")
    if not _native(state):
        spans = list(_spans(context_lens, q_start, q_lens, rows))
        y = _conv_ref(x.value(), conv, conv_state, spans, "silu")
        if q_lens is not None:
            y = y.to(dtype).float()
        o = _recur_ref(r, y, a.value(), None if b is None else b.value(), state, spans)
        if q_lens is not None:
            o = o.to(dtype)
        if parts:
            return gated_group_norm(o.reshape(T, inner), gate, gate_act, norm_w, parts, r.eps, dtype)
        o = o.float() / torch.sqrt(o.float().pow(2).mean(-1, keepdim=True) + r.eps) * norm_w
        return (o.reshape(T, inner) * ACTIVATIONS[gate_act][1](gate.value())).to(dtype)
    _check_conv(conv, conv_state)
    if state.dtype != torch.float32 or not state.is_contiguous() or tuple(state.shape[1:]) != r.state_shape:
        raise ValueError("state must be contiguous fp32 [slots, heads, vdim, dim_p]")
    for t in (r.rate, r.dt_bias, r.skip, norm_w):
        if t is not None and (t.dtype != torch.float32 or not t.is_contiguous()):
            raise TypeError("head_recurrence wants contiguous fp32 vectors")
    if x.width != conv.w.shape[1] or gate.width != inner or norm_w.numel() != (inner if parts else r.vdim):
        raise ValueError("sizes of channels, gate or norm do not fit")
    L, none = _lib.lib(), _lib.ProjArg(None, 0, 0, 1, 0)
    arg = _lib.HeadRecArg()
    arg.a, arg.b = a.arg(), none if b is None else b.arg()
    arg.rate, arg.dt_bias, arg.skip, arg.state = r.rate.data_ptr(), r.dt_bias.data_ptr(), _ptr(r.skip), state.data_ptr()
    arg.slot_ids, arg.context_lens = _ptr(rows), context_lens.data_ptr()
    arg.q_col, arg.k_col, arg.v_col, arg.gate_act = r.q_col, r.k_col, r.v_col, ACTIVATIONS[gate_act][0]
    arg.bf16, arg.batch, arg.tokens = 1 if dtype == torch.bfloat16 else 0, context_lens.shape[0], T
    arg.heads, arg.groups, arg.dim, arg.vdim = r.heads, r.groups, r.dim, r.vdim
    arg.q_scale, arg.eps, arg.unit_eps = float(r.q_scale), float(r.eps), UNIT_EPS
    if q_lens is None:
        if T != arg.batch:
            raise ValueError("a step has one token per sequence")
        out = torch.empty((T, inner), dtype=torch.float32 if parts else dtype, device=state.device)
        arg.x, arg.g, arg.conv_w, arg.conv_b = x.arg(), gate.arg(), conv.w.data_ptr(), _ptr(conv.bias)
        arg.conv_state, arg.taps, arg.channels = conv_state.data_ptr(), conv.taps, x.width
        arg.norm_w, arg.out = None if parts else norm_w.data_ptr(), out.data_ptr()
        _lib.check(L.nkb_head_rec_step(ctypes.byref(arg), _stream()), "nkb_head_rec_step")
        _count_launch()
        return gated_group_norm(out, gate, gate_act, norm_w, parts, r.eps, dtype) if parts else out
    y = short_conv(x, conv, conv_state, context_lens, q_start, q_lens, rows, dtype=dtype)
    out = torch.empty((T, inner), dtype=dtype, device=state.device)
    arg.x, arg.q_start, arg.q_lens, arg.out = Proj(y, 0, y.shape[1]).arg(), q_start.data_ptr(), q_lens.data_ptr(), out.data_ptr()
    _lib.check(L.nkb_head_rec_scan(ctypes.byref(arg), _stream()), "nkb_head_rec_scan")
    _count_launch()
    if parts:
        return gated_group_norm(out, gate, gate_act, norm_w, parts, r.eps, dtype)
    return gate_heads(out.view(T, r.heads, r.vdim), gate, gate_act, norm_w=norm_w, eps=r.eps)


def gated_group_norm(y: torch.Tensor, gate: Proj, act: str, norm_w: torch.Tensor, parts: int, eps: float,
                     dtype: torch.dtype = torch.bfloat16) -> torch.Tensor:
    """``norm_w * z / sqrt(mean(z^2) + eps)`` in `parts` equal parts of a row, z = y * act(gate), for y [T, W] -> [T, W]."""
    T, W = y.shape
    if W % parts or gate.width != W:
        raise ValueError("sizes of parts or gate do not fit")
    out = torch.empty((T, W), dtype=dtype, device=y.device)
    if not _native(y):
        z = (y.float() * ACTIVATIONS[act][1](gate.value())).reshape(T, parts, -1)
        z = z / torch.sqrt(z.pow(2).mean(-1, keepdim=True) + eps)
        return out.copy_((z.reshape(T, W) * norm_w).to(dtype))
    if norm_w.dtype != torch.float32 or not norm_w.is_contiguous() or not y.is_contiguous():
        raise TypeError("gated_group_norm wants contiguous rows and fp32 weights")
    rc = _lib.lib().nkb_gated_group_norm(y.data_ptr(), 1 if y.dtype == torch.bfloat16 else 0, _ref(gate), ACTIVATIONS[act][0],
                                         norm_w.data_ptr(), float(eps), out.data_ptr(), 1 if dtype == torch.bfloat16 else 0, T, W,
                                         parts, _stream())
    _lib.check(rc, "nkb_gated_group_norm")
    _count_launch()
    return out
