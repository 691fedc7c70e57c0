"""Operators of decoders whose layers mix attention and linear recurrences around an fp32 residual stream.

    gated_residual   embedding or residual + branches (gated, scaled, routed or normed, also through a norm of their sum; +
                     additions ahead of a repeated block, or an average with earlier results), and the norms of the
                     sum (group-wise RMS, layer norm, tanh, or a copy), in one launch
    gated_act        act(gate) * up, also with clamped operands or rows of a table as up; `activation` for act(x) alone
    gate_heads       scale * act(gate) * norm(head), the norm optional, one gate per element or per head
    hgrn2            linear attention with a per-channel forget gate; state in slots, fp32
    row_norm_append  queries and keys normed over all their heads, paged-cache append
    rope_norm_append biases, partial RoPE (half-split or interleaved, or none) and per-head norm of queries and keys,
                     paged-cache append
    maps_append      interleaved partial RoPE of queries / keys with several score maps, paged-cache append
    heads_attention  attention with several score maps over shared values (differential attention), score soft cap;
                     with one map plain grouped-query attention, also through a sliding window (with kept first
                     tokens), inside chunks, with sinks and with a distance term
    linear_simt      products on the CUDA cores: 32-bit models, operands TMA cannot describe

All of them take the projections they consume as `Proj` slices, so a decode-sized batch hands over split-K partial
sums and a prefill-sized one finished bf16 without a copy in between.  CUDA tensors run the kernels of
csrc/kernels/{gated_residual,post_residual,recurrent,attn_maps,attn_maps_prefill,gemm_simt}.cu; CPU tensors run the PyTorch
statement of the same op.
"""

from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import List, NamedTuple, Optional, Sequence, Tuple, Union

import torch
import torch.nn.functional as F

from . import _lib
from . import (ScoreMods, _count_launch, _decode_scratch, _gather_kv, _native, _ptr, _stream, flash_attn_prefill,
               paged_attn_decode, pick_kv_splits)

# name -> (kernel code, PyTorch function)
ACTIVATIONS = {"silu": (0, F.silu), "gelu_tanh": (1, lambda z: F.gelu(z, approximate="tanh")),
               "relu2": (2, lambda z: F.relu(z).square()), "tanh": (3, torch.tanh), "sigmoid": (4, torch.sigmoid),
               "none": (5, lambda z: z)}
CLAMPED = 6                  # of a gate and up pair (`gated_act`)
XIELU = 7                    # with two parameters (`Act`)


def xielu(z: torch.Tensor, a: float, b: float) -> torch.Tensor:
    return torch.where(z > 0, a * z * z, b * (torch.expm1(z) - z)) + z / 2


class Act(NamedTuple):
    """An activation with its parameters: "xielu" is a z^2 + z / 2 above zero and b (exp(z) - 1 - z) + z / 2 below."""
    name: str
    a: float = 0.0
    b: float = 0.0

    @staticmethod
    def of(act: Union[str, "Act"]) -> "Act":
        return act if isinstance(act, Act) else Act(act)

    @property
    def code(self) -> int:
        return XIELU if self.name == "xielu" else ACTIVATIONS[self.name][0]


def activate(z: torch.Tensor, act: Union[str, Act]) -> torch.Tensor:
    act = Act.of(act)
    return xielu(z, act.a, act.b) if act.name == "xielu" else ACTIVATIONS[act.name][1](z)


class Proj(NamedTuple):
    """Columns [col, col + width) of a projection's result: fp32 split-K partials [S, T, N], or bf16 / fp32 [T, N]."""
    t: torch.Tensor
    col: int
    width: int

    def value(self) -> torch.Tensor:
        """The finished slice in fp32, [T, width]."""
        x = self.t[..., self.col:self.col + self.width].float()
        return x.sum(0) if x.dim() == 3 else x

    def arg(self) -> _lib.ProjArg:
        t = self.t
        if t.stride(-1) != 1 or t.dtype not in (torch.float32, torch.bfloat16):
            raise ValueError("a projection slice needs unit column stride and fp32 or bf16 values")
        split = t.dim() == 3
        return _lib.ProjArg(t.data_ptr() + self.col * t.element_size(), t.stride(-2), t.stride(0) if split else 0,
                            t.shape[0] if split else 1, 1 if t.dtype == torch.bfloat16 else 0)


class Branch(NamedTuple):
    """One addend of a residual update: scale * y; with gate and bias, sigmoid(gate + bias) * y; with a gate of one column and no
    bias, scale * sigmoid(gate) * y; with pair_pos [T * k] and pair_w [T, k] (None with top_k = k: ones),
    scale * sum_j pair_w[t, j] * y[pair_pos[t * k + j]] (routed experts); with norm, scale * norm * y / sqrt(mean(y^2) + eps).
    shift (fp32 [width], a projection's bias) is added to y first, in plain and normed branches."""
    y: Proj
    gate: Optional[Proj] = None
    bias: Optional[torch.Tensor] = None
    scale: float = 1.0
    pair_pos: Optional[torch.Tensor] = None
    pair_w: Optional[torch.Tensor] = None
    top_k: int = 0
    norm: Optional[torch.Tensor] = None
    shift: Optional[torch.Tensor] = None

    @property
    def simple(self) -> bool:
        """Whether it is only scaled or normed."""
        return self.gate is None and self.pair_pos is None

    @property
    def chosen(self) -> int:
        return self.top_k if self.pair_w is None else self.pair_w.shape[1]

    def value(self, eps: float) -> torch.Tensor:
        if self.pair_pos is not None:
            pos = self.pair_pos.reshape(-1, self.chosen)
            rows = self.y.value()[pos.long().clamp(min=0)]
            w = (pos >= 0) if self.pair_w is None else self.pair_w * (pos >= 0)
            return self.scale * (rows * w[..., None]).sum(1)
        y = self.y.value() if self.shift is None else self.y.value() + self.shift
        if self.norm is not None:
            return self.scale * y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps) * self.norm
        if self.gate is not None:
            g = self.gate.value()
            return self.scale * y * torch.sigmoid(g if self.bias is None else g + self.bias)
        return self.scale * y

    def arg(self) -> _lib.BranchArg:
        none = _lib.ProjArg(None, 0, 0, 1, 0)
        token_gate = self.gate is not None and self.bias is None
        if token_gate and self.gate.width != 1:
            raise ValueError("a gate without bias has one column")
        if self.gate is not None and (self.pair_pos is not None or self.norm is not None or (not token_gate and self.scale != 1.0)):
            raise ValueError("a gated branch has neither routed rows nor a norm, and a scale only with one gate per token")
        return _lib.BranchArg(self.y.arg(), none if self.gate is None else self.gate.arg(), _ptr(self.bias),
                              _ptr(self.pair_pos), _ptr(self.pair_w), _ptr(self.norm),
                              0 if self.pair_pos is None else self.chosen, 1 if token_gate else 0, float(self.scale))


class Norm(NamedTuple):
    """What reads the residual: its RMS norm with a weight (a bare tensor means the same), with center its layer norm with
    weight and bias, with alpha tanh(alpha * x) * weight + bias (no mean or variance), without a weight the residual itself."""
    weight: Optional[torch.Tensor] = None
    bias: Optional[torch.Tensor] = None
    center: bool = False
    alpha: Optional[float] = None

    @property
    def kind(self) -> int:
        return 2 if self.weight is None else (3 if self.alpha is not None else 1 if self.center else 0)

    def value(self, x: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
        if self.weight is None:
            return x
        if self.alpha is not None:
            return torch.tanh(self.alpha * x) * self.weight + self.bias
        if self.center:
            d = x - x.mean(-1, keepdim=True)
            return d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + eps) * self.weight + self.bias
        return group_rmsnorm_ref(x, self.weight, groups, eps)

    def arg(self, out: Optional[torch.Tensor] = None) -> _lib.TanhNormArg:
        return _lib.TanhNormArg(_ptr(self.weight), _ptr(self.bias), float(self.alpha or 0.0), _ptr(out))


class History(NamedTuple):
    """Earlier results that a residual update averages with its own: sum_j coef[j] * rows[j] over j < past, + coef[past] * r.
    rows fp32 [n, T, W]; coef fp32 [past + 1]; store: r also goes to rows[past]."""
    rows: torch.Tensor
    past: int
    coef: torch.Tensor
    store: bool = True


def _ref(p: Proj):
    return ctypes.byref(p.arg())


def _ptr_array(ts: Sequence[Optional[torch.Tensor]]):
    return (ctypes.c_void_p * max(len(ts), 1))(*[_ptr(t) for t in ts])


def linear_simt(x: torch.Tensor, w: torch.Tensor, *, gated: bool = False, act: str = "silu",
                fp32_out: bool = False) -> torch.Tensor:
    """``x @ w.T`` with fp32 accumulation on the CUDA cores; x and w both fp32 or both bf16."""
    M, K = x.shape
    N = w.shape[0]
    f32 = x.dtype == torch.float32
    if x.dtype != w.dtype:
        raise TypeError(f"operands of different types: {x.dtype} and {w.dtype}")
    out = torch.empty((M, N), dtype=torch.float32 if f32 or fp32_out or gated else torch.bfloat16, device=x.device)
    rc = _lib.lib().nkb_gemm_simt(x.data_ptr(), 0 if f32 else 1, w.data_ptr(), 0 if f32 else 1, out.data_ptr(),
                                  0 if out.dtype == torch.float32 else 1, M, N, K, x.stride(0), w.stride(0), N, _stream())
    _lib.check(rc, "nkb_gemm_simt")
    _count_launch()
    if gated:
        return gated_act(Proj(out, 0, N // 2), Proj(out, N // 2, N // 2), act, dtype=x.dtype)
    return out


def group_rmsnorm_ref(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    y = x.float().reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    y = y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps)
    return y.reshape(x.shape) * w.float()


def gated_residual(x: Optional[torch.Tensor], branches: Sequence[Branch] = (), *,
                   ids: Optional[torch.Tensor] = None, table: Optional[torch.Tensor] = None, scale: float = 1.0,
                   add_mat: Optional[torch.Tensor] = None, add_row: Optional[torch.Tensor] = None,
                   norms: Sequence = (), groups: int = 1, eps: float = 1e-6, dtype: torch.dtype = torch.bfloat16,
                   post: Optional[Norm] = None, history: Optional[History] = None,
                   out: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, List[torch.Tensor]]:
    """One residual update of an fp32 stream and the norms that read it.

        r = x  (or table[ids] * scale)
        r += sum over branches (see `Branch`), with `post` (a tanh norm) its value of that sum;   r += add_mat;   r += add_row
        r = average with earlier results (see `History`)
        h_j = w_j * (r divided, in `groups` equal parts, by sqrt(mean(part^2) + eps)), or as `Norm` says (one kind per call)

    x [T, W] fp32; gate biases, add_row and the norm weights fp32 [W]; add_mat fp32 [T, W].  Returns (r, [h_j in `dtype`]), r in
    `out` when given."""
    branches = [b if isinstance(b, Branch) else Branch(*b) for b in branches]
    norms = [n if isinstance(n, Norm) else Norm(n) for n in norms]
    if len({n.kind for n in norms}) > 1:
        raise ValueError("the norms of one residual update are of one kind")
    if x is not None:
        rows, width = x.shape
        dev = x.device
    else:
        rows, width = ids.numel(), table.shape[1]
        dev = table.device
    r = out if out is not None else torch.empty((rows, width), dtype=torch.float32, device=dev)
    outs = [torch.empty((rows, width), dtype=dtype, device=dev) for _ in norms]
    if not _native(r):
        acc = x.clone() if x is not None else table[ids.long().clamp(0, table.shape[0] - 1)].float() * scale
        if branches:
            s = sum(b.value(eps) for b in branches)
            acc = acc + (s if post is None else post.value(s, 1, eps))
        if add_mat is not None:
            acc = acc + add_mat
        if add_row is not None:
            acc = acc + add_row
        if history is not None:
            if history.store:
                history.rows[history.past].copy_(acc)
            acc = acc * history.coef[-1] + torch.einsum("n,ntw->tw", history.coef[:-1], history.rows[:history.past])
        r.copy_(acc)
        for o, n in zip(outs, norms):
            o.copy_(n.value(acc, groups, eps).to(dtype))
        return r, outs
    if (post is not None or history is not None or any(n.kind == 3 for n in norms) or any(b.shift is not None for b in branches)
            or sum(b.norm is not None for b in branches) > 1):
        return _post_residual(x, branches, ids, table, scale, add_mat, add_row, norms, groups, eps, dtype, post, history, r, outs)
    weights, biases = [n.weight for n in norms], [n.bias for n in norms]
    for t in [x, add_mat, add_row, *weights, *biases, *[b.bias for b in branches], *[b.norm for b in branches]]:
        if t is not None and (t.dtype != torch.float32 or not t.is_contiguous()):
            raise TypeError("gated_residual wants contiguous fp32 residuals, biases and norm weights")
    n = len(branches)
    ba = (_lib.BranchArg * max(n, 1))(*[b.arg() for b in branches])
    rc = _lib.lib().nkb_gated_residual(
        _ptr(x), _ptr(ids), _ptr(table), 1 if table is not None and table.dtype == torch.bfloat16 else 0,
        table.shape[0] if table is not None else 0, float(scale), n, ba, _ptr(add_row), _ptr(add_mat), r.data_ptr(), len(outs),
        norms[0].kind if norms else 0, _ptr_array(weights), _ptr_array(biases), _ptr_array(outs),
        1 if dtype == torch.bfloat16 else 0, rows, width, int(groups), float(eps), _stream())
    _lib.check(rc, "nkb_gated_residual")
    _count_launch()
    return r, outs


def _post_residual(x, branches, ids, table, scale, add_mat, add_row, norms, groups, eps, dtype, post, history, r, outs):
    """The forms of `gated_residual` that csrc/kernels/post_residual.cu computes."""
    if len(branches) > 2 or not all(b.simple for b in branches):
        raise ValueError("a norm or an average after the sum takes at most two branches, scaled or normed")
    if post is not None and post.kind not in (2, 3):
        raise ValueError("the norm of the branches is a tanh norm")
    later = (norms and norms[0].kind in (0, 1)) or add_mat is not None or add_row is not None
    inner = [] if later else norms
    coef = None if history is None else history.coef
    for t in [x, coef, r, *[v for n in [post or Norm(), *inner] for v in (n.weight, n.bias)],
              *[v for b in branches for v in (b.norm, b.shift)]]:
        if t is not None and (t.dtype != torch.float32 or not t.is_contiguous()):
            raise TypeError("gated_residual wants contiguous fp32 residuals, biases and norm weights")
    a = _lib.PostResidualArg()
    a.x_in, a.ids, a.table, a.x_out = _ptr(x), _ptr(ids), _ptr(table), r.data_ptr()
    for i, b in enumerate(branches):
        a.br[i] = _lib.PostBranchArg(b.y.arg(), _ptr(b.shift), _ptr(b.norm), float(b.scale))
    a.post = (post or Norm()).arg()
    for i, (n, o) in enumerate(zip(inner, outs)):
        a.norm[i] = n.arg(o)
    if history is not None:
        rows = history.rows
        if rows.dtype != torch.float32 or not rows[0].is_contiguous() or coef.numel() != history.past + 1:
            raise ValueError("a history is fp32 rows and one coefficient per result")
        a.history, a.history_stride, a.past, a.coef = rows.data_ptr(), rows.stride(0), history.past, coef.data_ptr()
        a.result = rows[history.past].data_ptr() if history.store else None
    if table is not None:
        a.vocab, a.table_bf16 = table.shape[0], 1 if table.dtype == torch.bfloat16 else 0
    a.branches, a.norms, a.out_bf16 = len(branches), len(inner), 1 if dtype == torch.bfloat16 else 0
    a.rows, a.width = r.shape
    a.table_scale, a.eps = float(scale), float(eps)
    _lib.check(_lib.lib().nkb_post_residual(ctypes.byref(a), _stream()), "nkb_post_residual")
    _count_launch()
    if later:
        out, hs = gated_residual(r, add_mat=add_mat, add_row=add_row, norms=norms, groups=groups, eps=eps, dtype=dtype)
        return r.copy_(out), hs
    return r, outs


def gated_act(gate: Proj, up: Proj, act: str = "silu", dtype: torch.dtype = torch.bfloat16, *, limit: float = 0.0,
              alpha: float = 1.702, up_rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``act(gate) * up`` -> [T, width] in `dtype`; act "clamped": ``g * sigmoid(alpha * g) * (u + 1)`` with gate at most `limit`
    and up within +-limit.  up_rows [T] int32: up is a table, of which token t takes row up_rows[t]."""
    rows = gate.t.shape[-2]
    out = torch.empty((rows, gate.width), dtype=dtype, device=gate.t.device)
    if not _native(out):
        g, u = gate.value(), up.value()
        if up_rows is not None:
            u = u[up_rows.long().clamp(0, u.shape[0] - 1)]
        if act == "clamped":
            g = g.clamp(max=limit)
            return out.copy_((g * torch.sigmoid(alpha * g) * (u.clamp(-limit, limit) + 1)).to(dtype))
        return out.copy_((ACTIVATIONS[act][1](g) * u).to(dtype))
    kind = CLAMPED if act == "clamped" else ACTIVATIONS[act][0]
    rc = _lib.lib().nkb_gated_act(_ref(gate), _ref(up), out.data_ptr(), 1 if dtype == torch.bfloat16 else 0, rows,
                                  gate.width, kind, float(limit), float(alpha), _ptr(up_rows), up.t.shape[-2], _stream())
    _lib.check(rc, "nkb_gated_act")
    _count_launch()
    return out


def activation(x: Proj, act: Union[str, Act], dtype: torch.dtype = torch.bfloat16) -> torch.Tensor:
    """``act(x)`` -> [T, width] in `dtype`."""
    act = Act.of(act)
    rows = x.t.shape[-2]
    out = torch.empty((rows, x.width), dtype=dtype, device=x.t.device)
    if not _native(out):
        out.copy_(activate(x.value(), act).to(dtype))
        return out
    none = _lib.ProjArg(None, 0, 0, 1, 0)
    rc = _lib.lib().nkb_gated_act(_ref(x), ctypes.byref(none), out.data_ptr(), 1 if dtype == torch.bfloat16 else 0, rows,
                                  x.width, act.code, act.a, act.b, None, 0, _stream())
    _lib.check(rc, "nkb_gated_act")
    _count_launch()
    return out


def gate_heads(x: torch.Tensor, gate: Proj, act: str, *, norm_w: Optional[torch.Tensor] = None, eps: float = 1e-6,
               scale: float = 1.0, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``scale * act(gate) * x`` for heads x [T, H, n] (any strides of tokens and heads), gate [T, H * n] or, one per head,
    [T, H]; with norm_w (fp32, [n] shared by the
    heads or [H * n]) every head is first divided by its root mean square and multiplied by the weight.  Returns
    [T, H * n], written to `out` (a slice of columns) when given."""
    T, H, n = x.shape
    if out is None:
        out = torch.empty((T, H * n), dtype=x.dtype, device=x.device)
    if not _native(x):
        y = x.float()
        if norm_w is not None:
            y = y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps) * norm_w.float().reshape(-1, n)
        g = ACTIVATIONS[act][1](gate.value()).reshape(T, H, -1)
        out.copy_((scale * g * y).reshape(T, H * n).to(out.dtype))
        return out
    if x.stride(2) != 1 or out.stride(1) != 1 or x.dtype != out.dtype:
        raise ValueError("gate_heads wants unit column strides and one type")
    if gate.width not in (H, H * n):
        raise ValueError("one gate per element or per head")
    stride = 0 if norm_w is None or norm_w.numel() == n else n
    rc = _lib.lib().nkb_gate_heads(
        x.data_ptr(), 1 if x.dtype == torch.bfloat16 else 0, x.stride(0), x.stride(1), _ref(gate),
        1 if gate.width == H and n > 1 else 0, ACTIVATIONS[act][0], _ptr(norm_w), stride, float(eps), float(scale),
        out.data_ptr(), 1 if out.dtype == torch.bfloat16 else 0, out.stride(0), T, H, n, _stream())
    _lib.check(rc, "nkb_gate_heads")
    _count_launch()
    return out


# --------------------------------------------------------------------------- linear recurrence
def hgrn2_state_shape(heads: int, dim: int, vdim: int) -> Tuple[int, int, int]:
    """State of one sequence: [heads, vdim, dim rounded up to whole 16-byte pieces]."""
    return heads, vdim, (dim + 3) // 4 * 4


def hgrn2(q: Proj, f: Proj, v: Proj, f_bias: torch.Tensor, lower: torch.Tensor, norm_w: torch.Tensor,
          state: torch.Tensor, context_lens: torch.Tensor, *, heads: int, dim: int, vdim: int, eps: float,
          q_start: Optional[torch.Tensor] = None, q_lens: Optional[torch.Tensor] = None,
          rows: Optional[torch.Tensor] = None, dtype: torch.dtype = torch.bfloat16) -> torch.Tensor:
    """Gated linear recurrence over the new tokens of every sequence; returns the normed heads [T, heads * vdim].

        f = lower + (1 - lower) sigmoid(f + f_bias);   S <- diag(f) S + (1 - f) v^T;   o = S^T silu(q)
        o <- norm_w * o / sqrt(mean(o^2) + eps)   per head

    state [slots, heads, vdim, dim_p] fp32 is read and written in place at slot rows[b] (rows None: b).
    context_lens counts the new tokens; a sequence whose tokens are all new starts from a zero state, one with a
    negative length is skipped.  q_lens None: one new token per sequence (a decode step)."""
    T = q.t.shape[-2]
    out = torch.empty((T, heads * vdim), dtype=dtype, device=state.device)
    if not _native(state):
        qa = F.silu(q.value()).reshape(T, heads, dim)
        low = lower.float()
        fa = (low + (1 - low) * torch.sigmoid(f.value() + f_bias.float())).reshape(T, heads, dim)
        va = v.value().reshape(T, heads, vdim)
        o = torch.zeros((T, heads, vdim))
        for b in range(context_lens.shape[0]):
            n = 1 if q_lens is None else int(q_lens[b])
            t0 = b if q_lens is None else int(q_start[b])
            ctx, slot = int(context_lens[b]), b if rows is None else int(rows[b])
            if n <= 0 or ctx < n:
                continue
            S = torch.zeros((heads, vdim, dim)) if ctx == n else state[slot, :, :, :dim].clone()
            for t in range(t0, t0 + n):
                ft, vt = fa[t][:, None, :], va[t][:, :, None]
                S = ft * (S - vt) + vt
                o[t] = torch.einsum("hvd,hd->hv", S, qa[t])
            state[slot, :, :, :dim] = S
        if q_lens is not None and dtype == torch.bfloat16:
            o = o.to(dtype).float()
        o = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps) * norm_w.float()
        out.copy_(o.reshape(T, heads * vdim).to(dtype))
        return out
    if state.dtype != torch.float32 or not state.is_contiguous() or tuple(state.shape[1:]) != hgrn2_state_shape(
            heads, dim, vdim):
        raise ValueError("state must be contiguous fp32 [slots, heads, vdim, dim_p]")
    for t in (f_bias, lower, norm_w):
        if t.dtype != torch.float32 or not t.is_contiguous():
            raise TypeError("hgrn2 wants fp32 gate bias, lower bound and norm weight")
    L, bf = _lib.lib(), 1 if dtype == torch.bfloat16 else 0
    B = context_lens.shape[0]
    if q_lens is None:
        if T != B:
            raise ValueError("a step has one token per sequence")
        rc = L.nkb_hgrn2_step(_ref(q), _ref(f), _ref(v), f_bias.data_ptr(), lower.data_ptr(), state.data_ptr(),
                              _ptr(rows), context_lens.data_ptr(), out.data_ptr(), bf, B, heads, dim, vdim,
                              norm_w.data_ptr(), float(eps), _stream())
        _lib.check(rc, "nkb_hgrn2_step")
        _count_launch()
        return out
    scratch = torch.empty((T * L.nkb_hgrn2_scan_scratch(heads, dim, vdim),), dtype=torch.float32, device=state.device)
    rc = L.nkb_hgrn2_scan(_ref(q), _ref(f), _ref(v), f_bias.data_ptr(), lower.data_ptr(), state.data_ptr(), _ptr(rows),
                          q_start.data_ptr(), q_lens.data_ptr(), context_lens.data_ptr(), scratch.data_ptr(),
                          out.data_ptr(), bf, B, T, heads, dim, vdim, norm_w.data_ptr(), float(eps), _stream())
    _lib.check(rc, "nkb_hgrn2_scan")
    _count_launch(3)
    return out


# --------------------------------------------------------------------------- attention with score maps
def _tiled(n: int, sizes: Sequence[int]) -> int:
    for s in sizes:
        if n <= s:
            return s
    return (n + 1) // 2 * 2


@dataclass
class MapsSpec:
    """Sizes and constants of attention with `maps` score maps per head over shared values.  Two maps are combined as
    ``a0 - lam * a1``, root-mean-square normed over the head and multiplied by `out_scale`; softcap <= 0: none.
    dim_p / vdim_p are the padded sizes of queries / keys (per map) and values in the cache; the tiled bf16 kernels
    take 32 or 64 and 64 or 128, other sizes are only rounded to even and use the general kernel.  With one map the tiled
    kernels are those of plain attention, which take one size of 64 or 128 for both.  window > 0 (one map): a query sees
    itself and the window - 1 tokens before it, and the first keep_first ones.  chunk > 0 (one map): it sees the tokens of its own
    chunk of that many positions.  dist_a, dist_b (one map, fp32 [heads]): after the cap a score loses dist_a * ln(1 + dist_b *
    distance)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    maps: int = 1
    softcap: float = 0.0
    lam: float = 0.0
    out_scale: float = 1.0
    eps: float = 1e-6
    tiled: bool = True
    window: int = 0
    chunk: int = 0
    keep_first: int = 0
    dist_a: Optional[torch.Tensor] = None
    dist_b: Optional[torch.Tensor] = None

    @property
    def plain(self) -> bool:
        """Whether the kernels of plain attention serve this (one map, sizes they take)."""
        return self.tiled and self.maps == 1 and max(self.dim, self.vdim) <= 128

    @property
    def mods(self) -> ScoreMods:
        return ScoreMods(self.softcap, self.keep_first, self.dist_a, self.dist_b)

    @property
    def dim_p(self) -> int:
        if self.plain:
            return 64 if max(self.dim, self.vdim) <= 64 else 128
        return _tiled(self.dim, (32, 64) if self.tiled else ())

    @property
    def vdim_p(self) -> int:
        if self.plain:
            return self.dim_p
        return _tiled(self.vdim, (64, 128) if self.tiled else ())

    def arg(self) -> _lib.MapsArg:
        return _lib.MapsArg(self.maps, self.heads, self.kv_heads, self.dim, self.dim_p, self.vdim, self.vdim_p,
                            float(self.scale), float(self.softcap), float(self.lam), float(self.out_scale),
                            float(self.eps), int(self.window), int(self.chunk), None, 0, 0, 0, 0, 0, int(self.keep_first),
                            _ptr(self.dist_a), _ptr(self.dist_b))


def row_norm_append(spec: MapsSpec, q: Proj, k: Proj, v: Proj, q_norm: torch.Tensor, k_norm: torch.Tensor,
                    slots: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor) -> torch.Tensor:
    """RMS norms of a token's whole query and whole key projection (fp32 weights of those widths, spec.eps), keys and
    values written to their cache slots (negative slot: not stored); returns the queries [T, heads, dim_p]."""
    T = q.t.shape[-2]
    H, G, d, dp = spec.heads, spec.kv_heads, spec.dim, spec.dim_p
    bs = k_cache.shape[2]
    q_out = torch.empty((T, H, dp), dtype=k_cache.dtype, device=k_cache.device)
    if not _native(k_cache):
        def norm(x, w, n):
            x = x.value()
            x = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + spec.eps) * w
            return F.pad(x.reshape(T, n, d), (0, dp - d)).to(k_cache.dtype)

        q_out.copy_(norm(q, q_norm, H))
        sl = slots.long()
        keep = sl >= 0
        blk, off = sl[keep] // bs, sl[keep] % bs
        k_cache[blk, :, off] = norm(k, k_norm, G)[keep]
        v_cache[blk, :, off] = F.pad(v.value().reshape(T, G, spec.vdim), (0, spec.vdim_p - spec.vdim))[keep].to(v_cache.dtype)
        return q_out
    if q_norm.dtype != torch.float32 or k_norm.dtype != torch.float32:
        raise TypeError("row_norm_append wants fp32 norm weights")
    a = spec.arg()
    rc = _lib.lib().nkb_row_norm_append(ctypes.byref(a), _ref(q), _ref(k), _ref(v), q_norm.data_ptr(), k_norm.data_ptr(),
                                        slots.data_ptr(), q_out.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(),
                                        1 if k_cache.dtype == torch.bfloat16 else 0, T, bs, _stream())
    _lib.check(rc, "nkb_row_norm_append")
    _count_launch()
    return q_out


def half_rotate(x: torch.Tensor, cos_sin: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
    """x [T, n, d] fp32 with the first cos_sin.shape[1] dimensions rotated, dimension i paired with i + half."""
    n = cos_sin.shape[1] // 2
    cs = cos_sin[positions.long().clamp(0, cos_sin.shape[0] - 1)]
    c, s = cs[:, None, :n], cs[:, None, n:]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def pair_rotate(x: torch.Tensor, cos_sin: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
    """x [T, n, d] fp32 with the first cos_sin.shape[1] dimensions rotated, dimension 2i paired with 2i + 1."""
    n = cos_sin.shape[1] // 2
    cs = cos_sin[positions.long().clamp(0, cos_sin.shape[0] - 1)]
    c, s = cs[:, None, :n], cs[:, None, n:]
    u, v = x[..., :2 * n:2], x[..., 1:2 * n:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., 2 * n:]], -1)


def rope_norm_append(spec: MapsSpec, q: Proj, k: Optional[Proj], v: Optional[Proj], bias: Optional[torch.Tensor],
                     cos_sin: Optional[torch.Tensor], positions: torch.Tensor, slots: torch.Tensor, k_cache: torch.Tensor,
                     v_cache: torch.Tensor, norm: bool = True, interleaved: bool = False) -> torch.Tensor:
    """Add the biases (fp32 [q | k | v]), rotate the first cos_sin.shape[1] dimensions (cos_sin None: none) of every head of queries
    and keys (dimension i paired with i + half, interleaved: 2i with 2i + 1), with `norm` divide every head by
    sqrt(mean(head^2) + spec.eps), write keys and values to their cache slots (negative slot: not stored) and return the
    queries [T, heads, dim_p].  k and v None: only the queries."""
    T = q.t.shape[-2]
    H, G, d, dp = spec.heads, spec.kv_heads, spec.dim, spec.dim_p
    bs = k_cache.shape[2]
    q_out = torch.empty((T, H, dp), dtype=k_cache.dtype, device=k_cache.device)
    if not _native(k_cache):
        def head(x, n, first):
            x = x.value() if bias is None else x.value() + bias[first:first + x.width]
            x = x.reshape(T, n, d)
            if cos_sin is not None:
                x = (pair_rotate if interleaved else half_rotate)(x, cos_sin, positions)
            if norm:
                x = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + spec.eps)
            return F.pad(x, (0, dp - d)).to(k_cache.dtype)

        q_out.copy_(head(q, H, 0))
        if k is not None:
            sl = slots.long()
            keep = sl >= 0
            blk, off = sl[keep] // bs, sl[keep] % bs
            k_cache[blk, :, off] = head(k, G, q.width)[keep]
            x = v.value() if bias is None else v.value() + bias[q.width + k.width:]
            v_cache[blk, :, off] = F.pad(x.reshape(T, G, spec.vdim), (0, spec.vdim_p - spec.vdim))[keep].to(v_cache.dtype)
        return q_out
    for t in (bias, cos_sin):
        if t is not None and (t.dtype != torch.float32 or not t.is_contiguous()):
            raise TypeError("rope_norm_append wants fp32 biases and angles")
    a, none = spec.arg(), ctypes.byref(_lib.ProjArg(None, 0, 0, 1, 0))
    rc = _lib.lib().nkb_rope_norm_append(
        ctypes.byref(a), _ref(q), none if k is None else _ref(k), none if v is None else _ref(v), _ptr(bias),
        _ptr(cos_sin), *((0, 1) if cos_sin is None else (cos_sin.shape[1], cos_sin.shape[0])), positions.data_ptr(),
        slots.data_ptr(), 1 if norm else 0, 1 if interleaved else 0,
        q_out.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), 1 if k_cache.dtype == torch.bfloat16 else 0, T, bs, _stream())
    _lib.check(rc, "nkb_rope_norm_append")
    _count_launch()
    return q_out


def maps_append(spec: MapsSpec, q: Proj, k: Proj, v: Proj, cos_sin: torch.Tensor, positions: torch.Tensor,
                slots: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor) -> torch.Tensor:
    """Rotate queries and keys (pairs (2i, 2i + 1) of the first cos_sin.shape[1] dimensions of every map), write keys
    and values to their cache slots (negative slot: not stored), return the queries [T, heads, maps * dim_p]."""
    T = q.t.shape[-2]
    H, G, M, d, dp = spec.heads, spec.kv_heads, spec.maps, spec.dim, spec.dim_p
    bs = k_cache.shape[2]
    q_out = torch.empty((T, H, M * dp), dtype=k_cache.dtype, device=k_cache.device)
    rd = cos_sin.shape[1]
    if not _native(k_cache):
        cs = cos_sin[positions.long().clamp(0, cos_sin.shape[0] - 1)]
        c, s = cs[:, None, None, :rd // 2], cs[:, None, None, rd // 2:]

        def rot(x, n):
            x = F.pad(x.reshape(T, n, M, d), (0, dp - d))
            u, w = x[..., 0:rd:2].clone(), x[..., 1:rd:2].clone()
            x[..., 0:rd:2] = u * c - w * s
            x[..., 1:rd:2] = w * c + u * s
            return x.reshape(T, n, M * dp).to(k_cache.dtype)

        q_out.copy_(rot(q.value(), H))
        sl = slots.long()
        keep = sl >= 0
        blk, off = sl[keep] // bs, sl[keep] % bs
        k_cache[blk, :, off] = rot(k.value(), G)[keep]
        v_cache[blk, :, off] = F.pad(v.value().reshape(T, G, spec.vdim), (0, spec.vdim_p - spec.vdim))[keep].to(v_cache.dtype)
        return q_out
    a = spec.arg()
    rc = _lib.lib().nkb_maps_append(ctypes.byref(a), _ref(q), _ref(k), _ref(v), cos_sin.data_ptr(), rd, cos_sin.shape[0],
                                    positions.data_ptr(), slots.data_ptr(), q_out.data_ptr(), k_cache.data_ptr(),
                                    v_cache.data_ptr(), 1 if k_cache.dtype == torch.bfloat16 else 0, T, bs, _stream())
    _lib.check(rc, "nkb_maps_append")
    _count_launch()
    return q_out


def maps_attention(*args, **kw) -> torch.Tensor:
    """`heads_attention` with the heads side by side, [T, heads * vdim]."""
    return heads_attention(*args, **kw).flatten(1)


def heads_attention(spec: MapsSpec, q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                   block_table: torch.Tensor, context_lens: torch.Tensor, *, q_start: Optional[torch.Tensor] = None,
                   q_lens: Optional[torch.Tensor] = None, max_q_len: int = 1, num_splits: int = 0,
                   sinks: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention of the new tokens over the paged cache (which already holds them); returns the combined heads
    [T, heads, vdim] (strided when the cache's values are padded).  sinks [heads] fp32: logarithms of an addend of every
    softmax's denominator.  q_lens None: one new token per sequence (decode); otherwise sequence b owns rows
    q_start[b] .. q_start[b] + q_lens[b], the last of which sits at position context_lens[b] - 1."""
    T, H = q.shape[0], spec.heads
    bs = k_cache.shape[2]
    B = block_table.shape[0]
    if (spec.window > 0 or spec.chunk > 0 or sinks is not None or spec.dist_a is not None) and spec.maps != 1:
        raise ValueError("windows, chunks, sinks and distance terms are for one score map")
    if _native(k_cache) and spec.plain:
        qf = q.reshape(T, -1)
        if q_lens is None:
            o = paged_attn_decode(qf, k_cache, v_cache, block_table, context_lens, spec.scale, window=spec.window,
                                  chunk=spec.chunk, sinks=sinks, mods=spec.mods, num_splits=num_splits)
        else:
            o = flash_attn_prefill(qf, k_cache, v_cache, block_table, q_start, q_lens, context_lens, spec.scale,
                                   max_q_len=max_q_len, window=spec.window, chunk=spec.chunk, sinks=sinks, mods=spec.mods)
        return o.view(T, H, spec.vdim_p)[..., :spec.vdim]
    out = torch.empty((T, H, spec.vdim), dtype=k_cache.dtype, device=k_cache.device)
    if not _native(k_cache):
        M, dp = spec.maps, spec.dim_p
        res = torch.zeros((T, H, spec.vdim))
        rep = H // spec.kv_heads
        for b in range(B):
            n = 1 if q_lens is None else int(q_lens[b])
            t0 = b if q_lens is None else int(q_start[b])
            ctx = int(context_lens[b])
            if n <= 0 or ctx < n:
                continue
            k = _gather_kv(k_cache, block_table[b], ctx).float().reshape(ctx, spec.kv_heads, M, dp)
            v = _gather_kv(v_cache, block_table[b], ctx).float()[..., :spec.vdim]
            k, v = k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1)
            s = torch.einsum("qhmd,khmd->hmqk", q[t0:t0 + n].float().reshape(n, H, M, dp), k) * spec.scale
            pos = (ctx - n + torch.arange(n))[:, None]
            key = torch.arange(ctx)[None, :]
            s = spec.mods.apply(s, pos - key)
            vis = key <= pos
            if spec.window > 0:
                vis &= (key > pos - spec.window) | (key < spec.keep_first)
            if spec.chunk > 0:
                vis &= key >= pos - pos % spec.chunk
            s = s.masked_fill(~vis, float("-inf"))
            if sinks is not None:
                s = torch.cat([s, sinks.float()[:, None, None, None].expand(H, M, n, 1)], -1)
            a = torch.einsum("hmqk,khv->qhmv", s.softmax(-1)[..., :ctx], v)
            o = a[:, :, 0]
            if M == 2:
                o = o - spec.lam * a[:, :, 1]
                o = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + spec.eps) * spec.out_scale
            res[t0:t0 + n] = o
        out.copy_(res.to(out.dtype))
        return out
    L, a = _lib.lib(), spec.arg()
    a.sinks = _ptr(sinks)
    ref = ctypes.byref(a)
    bf = k_cache.dtype == torch.bfloat16
    common = (q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), block_table.data_ptr())
    rc = -5
    if bf and q_lens is None:
        group = H // spec.kv_heads
        if num_splits <= 0:
            num_splits = pick_kv_splits(B * spec.kv_heads * ((group + 7) // 8), block_table.shape[1])
        need = L.nkb_maps_decode_scratch_floats(ref, B, num_splits)
        scratch = _decode_scratch(q.device, need) if need else None
        rc = L.nkb_maps_attn_decode(ref, *common, context_lens.data_ptr(), out.data_ptr(), _ptr(scratch), B, bs,
                                    k_cache.shape[0], block_table.stride(0), num_splits, _stream())
    elif bf:
        rc = L.nkb_maps_attn_prefill(ref, *common, q_start.data_ptr(), q_lens.data_ptr(), context_lens.data_ptr(),
                                     out.data_ptr(), B, T, int(max_q_len), bs, k_cache.shape[0], block_table.stride(0),
                                     _stream())
    if rc == -5:
        if q_lens is None:
            q_start = torch.arange(B, dtype=torch.int32, device=q.device)
            q_lens = torch.ones((B,), dtype=torch.int32, device=q.device)
        rc = L.nkb_maps_attn_simple(ref, *common, q_start.data_ptr(), q_lens.data_ptr(), context_lens.data_ptr(),
                                    out.data_ptr(), 1 if bf else 0, B, T, bs, block_table.stride(0), _stream())
    _lib.check(rc, "maps_attention")
    _count_launch()
    return out
