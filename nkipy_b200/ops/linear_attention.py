"""Linear attention whose state decays per key channel, and the operators around it.

    token_mix         h + (previous token's h - h) * mu for several mu; the last h of a sequence is part of its state
    low_rank          W act(x) for a narrow x, in fp32
    linear_attention  the recurrence over the new tokens of every sequence with the norm and gate of its heads

CUDA tensors run csrc/kernels/linear_attn.cu; CPU tensors run the PyTorch statement of the same op.
"""

from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Tuple

import torch
import torch.nn.functional as F

from . import _lib
from . import _count_launch, _native, _ptr, _stream
from .mixers import ACTIVATIONS, Proj, _ref, activation

DECAYS = {"sigmoid_root": 0, "double_exp": 1}
_GEMM_ROWS = 128          # above: the low-rank product of a bf16 model is a tiled GEMM


@dataclass
class Decay:
    """Per-channel decay from the logit z = w act(x) + bias: "sigmoid_root" sigmoid(z)^(1 / tau), "double_exp"
    exp(-exp(z)).  x [T, rank] is the narrow projection, w [heads * dim, rank] of the model's type, bias fp32."""
    kind: str
    x: Proj
    w: torch.Tensor
    bias: torch.Tensor
    act: str = "none"
    tau: float = 1.0

    def value(self, z: torch.Tensor) -> torch.Tensor:
        if self.kind == "double_exp":
            return torch.exp(-torch.exp(z))
        return torch.exp(F.logsigmoid(z) / self.tau)


def token_mix(h: torch.Tensor, mu: torch.Tensor, state: torch.Tensor, context_lens: torch.Tensor, *,
              q_start: Optional[torch.Tensor] = None, q_lens: Optional[torch.Tensor] = None,
              rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out[m] = h + (h' - h) * mu[m] with h' the previous token's row of the same sequence (zeros before the first).

    h [T, W]; mu fp32 [M, W]; state fp32 [slots, W] holds the last row a sequence has seen and is read and written in
    place at slot rows[b] (rows None: b).  Sequences as in `linear_attention`.  Returns [M, T, W] in h's type."""
    T, W = h.shape
    M = mu.shape[0]
    out = torch.empty((M, T, W), dtype=h.dtype, device=h.device)
    B = context_lens.shape[0]
    if not _native(h):
        hf, prev = h.float(), torch.zeros((T, W))
        prev[1:] = hf[:-1]
        for b in range(B):
            n = 1 if q_lens is None else int(q_lens[b])
            t0 = b if q_lens is None else int(q_start[b])
            ctx, slot = int(context_lens[b]), b if rows is None else int(rows[b])
            if n <= 0:
                continue
            prev[t0] = state[slot] if ctx > n else 0.0
            if ctx >= n:
                state[slot] = hf[t0 + n - 1]
        out.copy_((hf + (prev - hf) * mu[:, None, :]).to(h.dtype))
        return out
    if (mu.dtype != torch.float32 or state.dtype != torch.float32 or not mu.is_contiguous() or not state.is_contiguous()
            or not h.is_contiguous() or tuple(state.shape[1:]) != (W,)):
        raise TypeError("token_mix wants contiguous rows, fp32 mixes and state")
    rc = _lib.lib().nkb_token_mix(h.data_ptr(), 1 if h.dtype == torch.bfloat16 else 0, mu.data_ptr(), state.data_ptr(),
                                  _ptr(rows), _ptr(q_start), _ptr(q_lens), context_lens.data_ptr(), out.data_ptr(), B, T, W,
                                  M, _stream())
    _lib.check(rc, "nkb_token_mix")
    _count_launch()
    return out


def low_rank(x: Proj, w: torch.Tensor, act: str = "none") -> torch.Tensor:
    """``act(x) @ w.T`` in fp32 [T, N], w [N, rank]."""
    T = x.t.shape[-2]
    N, rank = w.shape
    if x.width != rank:
        raise ValueError(f"low-rank input of width {x.width}, weight {tuple(w.shape)}")
    if not _native(w):
        return ACTIVATIONS[act][1](x.value()) @ w.float().T
    if T > _GEMM_ROWS and w.dtype == torch.bfloat16 and rank % 8 == 0:
        from . import linear

        a = activation(x, act)
        return linear(a, w, swap=False, fp32_out=True)
    out = torch.empty((T, N), dtype=torch.float32, device=w.device)
    rc = _lib.lib().nkb_low_rank(_ref(x), ACTIVATIONS[act][0], w.data_ptr(), 1 if w.dtype == torch.bfloat16 else 0,
                                 out.data_ptr(), T, rank, N, _stream())
    _lib.check(rc, "nkb_low_rank")
    _count_launch()
    return out


def linear_state_shape(heads: int, dim: int, vdim: int) -> Tuple[int, int, int]:
    """State of one sequence: [heads, vdim, dim rounded up to whole 16-byte pieces]."""
    return heads, vdim, (dim + 3) // 4 * 4


def linear_attention(q: Proj, k: Proj, v: Proj, decay: Decay, gate: Proj, norm_w: torch.Tensor, state: torch.Tensor,
                     context_lens: torch.Tensor, *, heads: int, dim: int, vdim: int, eps: float, q_scale: float = 1.0,
                     bonus: Optional[torch.Tensor] = None, scale: float = 1.0, gate_act: str = "silu",
                     q_start: Optional[torch.Tensor] = None, q_lens: Optional[torch.Tensor] = None,
                     rows: Optional[torch.Tensor] = None, dtype: torch.dtype = torch.bfloat16,
                     out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Per head S <- diag(decay) S + k v^T over the new tokens of every sequence, read with q_scale * q after the update, or
    with `bonus` (fp32 [heads * dim]) before it, the current token then entering through diag(bonus) k v^T.  Returns

        scale * gate_act(gate) * norm_w * o / sqrt(mean(o^2) + eps)      [T, heads * vdim]

    (norm_w fp32, [vdim] shared by the heads or [heads * vdim]), written to `out` (a slice of columns) when given.

    state [slots, heads, vdim, dim_p] fp32 is read and written in place at slot rows[b] (rows None: b).
    context_lens counts the new tokens; a sequence whose tokens are all new starts from a zero state, one with a
    negative length is skipped.  q_lens None: one new token per sequence (a decode step)."""
    T = q.t.shape[-2]
    if out is None:
        out = torch.empty((T, heads * vdim), dtype=dtype, device=state.device)
    if not _native(state):
        z = low_rank(decay.x, decay.w, decay.act) + decay.bias
        a = decay.value(z).reshape(T, heads, dim)
        qa, ka = (p.value().reshape(T, heads, dim) for p in (q, k))
        va = v.value().reshape(T, heads, vdim)
        u = bonus.reshape(heads, 1, dim) if bonus is not None else None
        o = torch.zeros((T, heads, vdim))
        for b in range(context_lens.shape[0]):
            n = 1 if q_lens is None else int(q_lens[b])
            t0 = b if q_lens is None else int(q_start[b])
            ctx, slot = int(context_lens[b]), b if rows is None else int(rows[b])
            if n <= 0 or ctx < n:
                continue
            S = torch.zeros((heads, vdim, dim)) if ctx == n else state[slot, :, :, :dim].clone()
            for t in range(t0, t0 + n):
                kv = ka[t][:, None, :] * va[t][:, :, None]
                if u is not None:
                    o[t] = torch.einsum("hvd,hd->hv", S + u * kv, qa[t])
                S = a[t][:, None, :] * S + kv
                if u is None:
                    o[t] = torch.einsum("hvd,hd->hv", S, qa[t])
            state[slot, :, :, :dim] = S
        o = o * q_scale
        if q_lens is not None and dtype == torch.bfloat16:
            o = o.to(dtype).float()
        o = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps) * norm_w.reshape(-1, vdim)
        out.copy_((scale * ACTIVATIONS[gate_act][1](gate.value()) * o.reshape(T, -1)).to(out.dtype))
        return out
    if state.dtype != torch.float32 or not state.is_contiguous() or tuple(state.shape[1:]) != linear_state_shape(
            heads, dim, vdim):
        raise ValueError("state must be contiguous fp32 [slots, heads, vdim, dim_p]")
    for t in (decay.bias, norm_w, bonus):
        if t is not None and (t.dtype != torch.float32 or not t.is_contiguous()):
            raise TypeError("linear_attention wants fp32 decay bias, bonus and norm weight")
    if out.stride(1) != 1 or out.dtype != dtype or not decay.w.is_contiguous():
        raise ValueError("linear_attention wants unit column stride and contiguous decay weights")
    a = _lib.LinAttnArg()
    a.q, a.k, a.v, a.g = q.arg(), k.arg(), v.arg(), gate.arg()
    a.z_bias, a.bonus, a.norm_w, a.state = decay.bias.data_ptr(), _ptr(bonus), norm_w.data_ptr(), state.data_ptr()
    a.slot_ids, a.context_lens = _ptr(rows), context_lens.data_ptr()
    a.out, a.out_ld = out.data_ptr(), out.stride(0)
    a.decay, a.inv_tau, a.z_act = DECAYS[decay.kind], 1.0 / decay.tau, ACTIVATIONS[decay.act][0]
    a.norm_stride = 0 if norm_w.numel() == vdim else vdim
    a.gate_act, a.bf16 = ACTIVATIONS[gate_act][0], 1 if dtype == torch.bfloat16 else 0
    a.batch, a.tokens, a.heads, a.dim, a.vdim = context_lens.shape[0], T, heads, dim, vdim
    a.q_scale, a.out_scale, a.eps = float(q_scale), float(scale), float(eps)
    L = _lib.lib()
    if q_lens is None:
        if T != a.batch:
            raise ValueError("a step has one token per sequence")
        a.z, a.w2, a.w2_bf16, a.rank = decay.x.arg(), decay.w.data_ptr(), 1 if decay.w.dtype == torch.bfloat16 else 0, decay.w.shape[1]
        _lib.check(L.nkb_linattn_step(ctypes.byref(a), _stream()), "nkb_linattn_step")
        _count_launch()
        return out
    z = low_rank(decay.x, decay.w, decay.act)
    raw = torch.empty((T, heads * vdim), dtype=dtype, device=state.device)
    a.z, a.q_start, a.q_lens, a.heads_out = Proj(z, 0, z.shape[1]).arg(), q_start.data_ptr(), q_lens.data_ptr(), raw.data_ptr()
    _lib.check(L.nkb_linattn_scan(ctypes.byref(a), _stream()), "nkb_linattn_scan")
    _count_launch(2)
    return out
