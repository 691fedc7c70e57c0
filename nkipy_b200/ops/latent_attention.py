"""Operators of latent attention: all heads share one cached row per token, a normed latent and a rotated key part.

    latent_append     norms of the two down projections, rotation of the key part, cache row
    latent_queries    up-projected queries split and rotated
    latent_attention  new tokens against the cached rows themselves (queries folded through the keys' up projection)
    latent_gather     cached rows of whole pages, as operands of the keys' and values' up projections
    latent_prefill    new tokens against keys and values expanded from those rows

CUDA tensors run csrc/kernels/latent_attn.cu and, for expanded keys, attn_prefill.cu (32-bit models and sizes the tensor-core
kernel does not take: the general kernel of attn_maps.cu); CPU tensors run the PyTorch statement of the same op.
"""

from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Tuple

import torch
import torch.nn.functional as F

from . import _lib
from . import _count_launch, _gather_kv, _native, _ptr, _stream
from .mixers import Proj, _ref

# (64-column slabs of a cached row, of its latent) the tensor-core kernel is built for
_SHAPES = ((2, 1), (3, 2), (5, 4), (9, 8))


@dataclass
class LatentSpec:
    """Sizes and constants; window > 0: a query sees itself and the window - 1 tokens before it.  `row` is the padded size of a
    cached row [latent, rotated part, zeros]."""
    heads: int
    dim: int
    rot: int
    vdim: int
    rank: int
    q_rank: int
    scale: float
    window: int = 0
    eps: float = 1e-6
    tiled: bool = True

    @property
    def row(self) -> int:
        if self.tiled:
            for ns, vs in _SHAPES:
                if self.rank <= 64 * vs and self.rank + self.rot <= 64 * ns:
                    return 64 * ns
        return (self.rank + self.rot + 7) // 8 * 8

    @property
    def slabs(self) -> Optional[Tuple[int, int]]:
        """64-column slabs of expanded queries and keys (the last one rotated) and of values in the prefill kernel; None for
        sizes it does not take."""
        if not self.tiled or self.dim > 128 or self.rot > 64 or self.vdim > 128 or (self.dim | self.vdim | self.rank) % 8:
            return None
        return (2, 1 if self.vdim <= 64 else 2) if self.dim <= 64 else (3, 2)

    def arg(self) -> _lib.LatentArg:
        return _lib.LatentArg(self.heads, self.dim, self.rot, self.rank, self.q_rank, self.row, float(self.eps),
                              float(self.scale), int(self.window), None, 0, 0, 0, 0)


def _pick_splits(units: int, pages: int, sms: int = 148) -> int:
    """CTAs (1, 2, 4 or 8) that share a token's pages: as many as leave each four pages while every SM has at most one."""
    s = 1
    while s < 8 and 2 * s * units <= sms and pages >= 8 * s:
        s *= 2
    return s


def pair_rotate(x: torch.Tensor, cos_sin: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
    """x [T, n, d] fp32 with dimensions 2i and 2i + 1 rotated."""
    n = cos_sin.shape[1] // 2
    cs = cos_sin[positions.long().clamp(0, cos_sin.shape[0] - 1)]
    c, s = cs[:, None, :n], cs[:, None, n:]
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)


def latent_append(spec: LatentSpec, q: Proj, kv: Proj, q_norm: torch.Tensor, kv_norm: torch.Tensor, cos_sin: torch.Tensor,
                  positions: torch.Tensor, slots: torch.Tensor, cache: torch.Tensor) -> torch.Tensor:
    """RMS norms (fp32 weights) of the query latent q [T, q_rank] and of the first `rank` columns of kv, rotation of its last
    `rot` columns; the latter two go to the cache [blocks, 1, 32, row] (negative slot: not stored).  Returns the query latent
    in the cache's type."""
    T, bs = q.t.shape[-2], cache.shape[2]
    out = torch.empty((T, spec.q_rank), dtype=cache.dtype, device=cache.device)
    if not _native(cache):
        norm = lambda x, w: x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + spec.eps) * w
        out.copy_(norm(q.value(), q_norm))
        x = kv.value()
        r = pair_rotate(x[:, None, spec.rank:], cos_sin, positions)[:, 0]
        row = F.pad(torch.cat([norm(x[:, :spec.rank], kv_norm), r], -1), (0, spec.row - spec.rank - spec.rot))
        sl = slots.long()
        keep = sl >= 0
        cache[sl[keep] // bs, 0, sl[keep] % bs] = row[keep].to(cache.dtype)
        return out
    for t in (q_norm, kv_norm, cos_sin):
        if t.dtype != torch.float32 or not t.is_contiguous():
            raise TypeError("latent_append wants fp32 norm weights and angles")
    a = spec.arg()
    rc = _lib.lib().nkb_latent_append(ctypes.byref(a), _ref(q), _ref(kv), q_norm.data_ptr(), kv_norm.data_ptr(),
                                      cos_sin.data_ptr(), cos_sin.shape[0], positions.data_ptr(), slots.data_ptr(),
                                      out.data_ptr(), cache.data_ptr(), 1 if cache.dtype == torch.bfloat16 else 0, T, bs,
                                      _stream())
    _lib.check(rc, "nkb_latent_append")
    _count_launch()
    return out


def latent_queries(spec: LatentSpec, q: Proj, cos_sin: torch.Tensor, positions: torch.Tensor, plain: torch.Tensor,
                   rotated: torch.Tensor) -> None:
    """Split the queries [T, heads * (dim + rot)] into `plain` [T, heads, >= dim] and, rotated, `rotated` [T, heads, >= rot];
    both are views with any strides of tokens and heads, filled up with zeros."""
    T, H = q.t.shape[-2], spec.heads
    if not _native(plain):
        x = q.value().reshape(T, H, spec.dim + spec.rot)
        plain.copy_(F.pad(x[..., :spec.dim], (0, plain.shape[2] - spec.dim)))
        rotated.copy_(F.pad(pair_rotate(x[..., spec.dim:], cos_sin, positions), (0, rotated.shape[2] - spec.rot)))
        return
    if plain.stride(2) != 1 or rotated.stride(2) != 1 or plain.dtype != rotated.dtype:
        raise ValueError("latent_queries wants unit column strides and one type")
    a = spec.arg()
    rc = _lib.lib().nkb_latent_queries(
        ctypes.byref(a), _ref(q), cos_sin.data_ptr(), cos_sin.shape[0], positions.data_ptr(), plain.data_ptr(),
        plain.stride(0), plain.stride(1), plain.shape[2], rotated.data_ptr(), rotated.stride(0), rotated.stride(1),
        rotated.shape[2], 1 if plain.dtype == torch.bfloat16 else 0, T, _stream())
    _lib.check(rc, "nkb_latent_queries")
    _count_launch()


def latent_gather(spec: LatentSpec, cache: torch.Tensor, pages: torch.Tensor, rot_ld: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """Rows of the given cache pages (int32 block numbers): latents [32 P, rank] and rotated parts [32 P, rot_ld] (columns past
    `rot` unspecified)."""
    bs, P = cache.shape[2], pages.shape[0]
    c = torch.empty((P * bs, spec.rank), dtype=cache.dtype, device=cache.device)
    r = torch.empty((P * bs, rot_ld), dtype=cache.dtype, device=cache.device)
    if not _native(cache):
        rows = cache[pages.long(), 0].reshape(P * bs, -1)
        c.copy_(rows[:, :spec.rank])
        r[:, :spec.rot] = rows[:, spec.rank:spec.rank + spec.rot]
        return c, r
    rc = _lib.lib().nkb_latent_gather(cache.data_ptr(), pages.data_ptr(), P, spec.row, spec.rank, spec.rot, rot_ld,
                                      c.data_ptr(), r.data_ptr(), 1 if cache.dtype == torch.bfloat16 else 0, bs, _stream())
    _lib.check(rc, "nkb_latent_gather")
    _count_launch()
    return c, r


def latent_attention(spec: LatentSpec, q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor,
                     context_lens: torch.Tensor, *, q_start: Optional[torch.Tensor] = None,
                     q_lens: Optional[torch.Tensor] = None, sinks: Optional[torch.Tensor] = None,
                     num_splits: int = 0) -> torch.Tensor:
    """Causal attention of queries over cached rows: q [heads, T, row] (the part against the latent, the rotated part, zeros)
    -> mixtures of latents [heads, T, rank].  sinks [heads] fp32: logarithms of an addend of every softmax's denominator.
    q_lens None: one new token per sequence; otherwise sequence b owns rows q_start[b] .. q_start[b] + q_lens[b], the last of
    which sits at position context_lens[b] - 1."""
    H, T, row = q.shape
    B, bs = block_table.shape[0], cache.shape[2]
    out = torch.empty((H, T, spec.rank), dtype=cache.dtype, device=cache.device)
    if not _native(cache):
        out.zero_()
        for b in range(B):
            n = 1 if q_lens is None else int(q_lens[b])
            t0 = b if q_lens is None else int(q_start[b])
            ctx = int(context_lens[b])
            if n <= 0 or ctx < n:
                continue
            k = _gather_kv(cache, block_table[b], ctx)[:, 0].float()
            s = torch.einsum("htd,kd->htk", q[:, t0:t0 + n].float(), k) * spec.scale
            pos = (ctx - n + torch.arange(n))[:, None]
            vis = torch.arange(ctx)[None, :] <= pos
            if spec.window > 0:
                vis &= torch.arange(ctx)[None, :] > pos - spec.window
            s = s.masked_fill(~vis, float("-inf"))
            if sinks is not None:
                s = torch.cat([s, sinks.float()[:, None, None].expand(H, n, 1)], -1)
            out[:, t0:t0 + n] = (s.softmax(-1)[..., :ctx] @ k[:, :spec.rank]).to(out.dtype)
        return out
    if row != spec.row or not q.is_contiguous() or q.dtype != cache.dtype:
        raise ValueError("latent_attention wants contiguous queries of the cache's row size and type")
    L, bf = _lib.lib(), cache.dtype == torch.bfloat16
    rc = -5
    if bf:
        a = spec.arg()
        a.sinks, a.q_token, a.q_head, a.o_token, a.o_head = _ptr(sinks), row, T * row, spec.rank, T * spec.rank
        if num_splits <= 0:
            pages = block_table.shape[1] if spec.window <= 0 else min(block_table.shape[1], spec.window // bs + 2)
            num_splits = _pick_splits(T * ((H + 31) // 32), pages)
        rc = L.nkb_latent_attn(ctypes.byref(a), q.data_ptr(), cache.data_ptr(), block_table.data_ptr(), _ptr(q_start),
                               _ptr(q_lens), context_lens.data_ptr(), out.data_ptr(), B, T, bs, cache.shape[0],
                               block_table.stride(0), num_splits, _stream())
    if rc == -5:
        if q_lens is None:
            q_start = torch.arange(B, dtype=torch.int32, device=q.device)
            q_lens = torch.ones((B,), dtype=torch.int32, device=q.device)
        m = _lib.MapsArg(1, H, 1, spec.rank + spec.rot, row, spec.rank, spec.rank, float(spec.scale), 0.0, 0.0, 1.0,
                         float(spec.eps), int(spec.window), 0, _ptr(sinks), row, T * row, spec.rank, T * spec.rank, row)
        rc = L.nkb_maps_attn_simple(ctypes.byref(m), q.data_ptr(), cache.data_ptr(), cache.data_ptr(), block_table.data_ptr(),
                                    q_start.data_ptr(), q_lens.data_ptr(), context_lens.data_ptr(), out.data_ptr(),
                                    1 if bf else 0, B, T, bs, block_table.stride(0), _stream())
    _lib.check(rc, "latent_attention")
    _count_launch()
    return out


def latent_prefill(spec: LatentSpec, q: torch.Tensor, kv: torch.Tensor, rotated: torch.Tensor, kv_base: torch.Tensor,
                   q_start: torch.Tensor, q_lens: torch.Tensor, context_lens: torch.Tensor, max_q_len: int,
                   sinks: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention over expanded rows: kv [rows, heads * dim | heads * vdim] and rotated [rows, >= rot] hold position j of
    sequence b in row kv_base[b] + j; q [T, heads, 64 nk] has a head's unrotated part in front and its rotated part in the
    last 64 columns.  Returns [T, heads, vdim] (strided)."""
    T, H = q.shape[0], spec.heads
    nk, nv = spec.slabs
    out = torch.empty((T, H, 64 * nv), dtype=q.dtype, device=q.device)
    if not _native(q):
        out.zero_()
        split = H * spec.dim
        for b in range(q_lens.shape[0]):
            n, t0, ctx, base = int(q_lens[b]), int(q_start[b]), int(context_lens[b]), int(kv_base[b])
            lo = max(0, ctx - n - spec.window + 1) if spec.window > 0 else 0
            rows = slice(base + lo, base + ctx)
            x = q[t0:t0 + n].float()
            k = kv[rows, :split].float().reshape(-1, H, spec.dim)
            v = kv[rows, split:split + H * spec.vdim].float().reshape(-1, H, spec.vdim)
            s = torch.einsum("qhd,khd->hqk", x[..., :spec.dim], k)
            s = (s + torch.einsum("qhd,kd->hqk", x[..., -64:][..., :spec.rot], rotated[rows, :spec.rot].float())) * spec.scale
            i, j = (ctx - n + torch.arange(n))[:, None], torch.arange(lo, ctx)[None, :]
            vis = j <= i
            if spec.window > 0:
                vis &= j > i - spec.window
            s = s.masked_fill(~vis, float("-inf"))
            if sinks is not None:
                s = torch.cat([s, sinks.float()[:, None, None].expand(H, n, 1)], -1)
            out[t0:t0 + n, :, :spec.vdim] = torch.einsum("hqk,khn->qhn", s.softmax(-1)[..., :ctx - lo], v).to(out.dtype)
        return out[..., :spec.vdim]
    if not q.is_contiguous() or q.shape[2] != 64 * nk or q.dtype != torch.bfloat16 or kv.dtype != torch.bfloat16:
        raise ValueError("latent_prefill wants contiguous bf16 queries of whole slabs")
    rc = _lib.lib().nkb_latent_prefill(
        q.data_ptr(), kv.data_ptr(), rotated.data_ptr(), q_start.data_ptr(), q_lens.data_ptr(), context_lens.data_ptr(),
        kv_base.data_ptr(), out.data_ptr(), q_lens.shape[0], T, int(max_q_len), kv.shape[0], H, spec.dim, spec.rot, spec.vdim,
        kv.stride(0), rotated.stride(0), nk, nv, float(spec.scale), int(spec.window), _ptr(sinks), _stream())
    _lib.check(rc, "nkb_latent_prefill")
    _count_launch()
    return out[..., :spec.vdim]
