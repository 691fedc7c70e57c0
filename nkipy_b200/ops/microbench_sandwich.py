"""Micro-benchmark cases of layers normed on both sides, recurrences with one decay per head and attention with modified scores, at
the shapes of the like kernels in microbench_mixers.py."""
from __future__ import annotations

import torch

from . import linear
from .head_recurrence import HeadRecurrence, ShortConv, gated_group_norm, head_recurrence, short_conv
from .microbench_mixers import G, H, V, W, _bf16, _i32
from .mixers import Act, Branch, History, MapsSpec, Norm, Proj, activation, gated_residual, heads_attention, rope_norm_append

GROUPS = 8


def _result(name, args, timer, fns, bytes, flops, **shape):
    return dict(case=name, us=timer(fns, args.iters, args.warmup, not args.no_graph), bytes=bytes, flops=flops, shape=shape)


def _vec(n, value=None):
    return torch.randn(n, device="cuda") if value is None else torch.full((n,), value, device="cuda")


def _rec(T, delta):
    """(arguments of a recurrence over 32 heads of 128 x 128, recurrence, channels)."""
    groups = H if delta else GROUPS
    C = W + 2 * groups * V
    y = _bf16(T, C + W + 64)
    q, k, v = (0, groups * V, 2 * groups * V) if delta else (W + groups * V, W, 0)
    rec = HeadRecurrence(H, groups, V, V, q, k, v, _vec(H, 0.1), _vec(H), delta, V ** -0.5, None if delta else _vec(H), 1e-5)
    conv = ShortConv(torch.randn(4, C, device="cuda") / 2, None if delta else _vec(C))
    return (Proj(y, 0, C), conv, Proj(y, C + W, H), Proj(y, C + W + 32, H) if delta else None, Proj(y, C, W),
            _vec(V if delta else W, 1.0)), rec, C


def rec_step(delta):
    def case(args, timer, sets_for):
        B = 64
        state_bytes = B * H * V * V * 4
        sets = sets_for(2 * state_bytes, args.sets)
        a, rec, C = _rec(B, delta)
        states = [torch.randn(B, *rec.state_shape, device="cuda") for _ in range(sets)]
        ring, lens = torch.randn(B, 4, C, device="cuda"), torch.full((B,), 77, device="cuda", dtype=torch.int32)
        fns = [lambda st=st: head_recurrence(rec, *a, st, ring, lens, parts=0 if delta else GROUPS) for st in states]
        return _result("delta-step" if delta else "ssd-step", args, timer, fns, 2 * state_bytes + B * (C * 18 + W * 4),
                       B * H * V * V * 8.0, batch=B, heads=H, dim=V, vdim=V, taps=4, sets=sets)
    return case


def rec_scan(delta):
    def case(args, timer, sets_for):
        B, S = args.batch or 8, args.seq or 2048
        a, rec, C = _rec(B * S, delta)
        state, ring = torch.zeros(B, *rec.state_shape, device="cuda"), torch.zeros(B, 4, C, device="cuda")
        start, lens, rows = _i32(range(B)) * S, torch.full((B,), S, device="cuda", dtype=torch.int32), _i32(range(B))
        fns = [lambda: head_recurrence(rec, *a, state, ring, lens, parts=0 if delta else GROUPS, q_start=start, q_lens=lens,
                                       rows=rows)]
        # operations: decay, write, and two products (delta rule) or one with the state
        return _result("delta-scan" if delta else "ssd-scan", args, timer, fns, B * S * (3 * C + 4 * W) * 2,
                       B * S * H * V * V * (7.0 if delta else 5.0), batch=B, seq=S, heads=H, dim=V, vdim=V, taps=4)
    return case


def conv(args, timer, sets_for):
    B, S = args.batch or 8, args.seq or 2048
    a, _, C = _rec(B * S, True)
    ring, start, lens = torch.zeros(B, 4, C, device="cuda"), _i32(range(B)) * S, torch.full((B,), S, device="cuda", dtype=torch.int32)
    fns = [lambda: short_conv(a[0], a[1], ring, lens, start, lens)]
    return _result("short-conv-16384", args, timer, fns, B * S * C * 4, 0.0, tokens=B * S, channels=C, taps=4)


def group_norm(tokens, splits):
    def case(args, timer, sets_for):
        y = torch.randn(tokens, W, device="cuda") if splits else _bf16(tokens, W)
        z, w = torch.randn(splits, tokens, W, device="cuda") if splits else _bf16(tokens, W), _vec(W, 1.0)
        fns = [lambda: gated_group_norm(y, Proj(z, 0, W), "silu", w, GROUPS, 1e-5)]
        return _result(f"group-norm-{tokens}", args, timer, fns, tokens * W * ((4 + 4 * splits if splits else 4) + 2), 0.0, tokens=tokens,
                       width=W, parts=GROUPS, splits=splits)
    return case


def _attn_spec(kind):
    if kind == "capped":
        return MapsSpec(H, G, V, V, V ** -0.5, softcap=30.0), _vec(H)
    return MapsSpec(H, G, V, V, V ** -0.5, softcap=30.0, window=1024, keep_first=4, dist_a=_vec(H).abs(), dist_b=_vec(H).abs()), None


def attn_prefill(kind, qscale=1.0):
    def case(args, timer, sets_for):
        B, S = args.batch or 8, args.seq or 2048
        s, sinks = _attn_spec(kind)
        nb = B * S // 32
        k, v, q = _bf16(nb, G, 32, V), _bf16(nb, G, 32, V), _bf16(B * S, H, V, scale=qscale)
        table = _i32(range(nb)).reshape(B, S // 32)
        start, lens = _i32(range(B)) * S, torch.full((B,), S, device="cuda", dtype=torch.int32)
        fns = [lambda: heads_attention(s, q, k, v, table, lens, q_start=start, q_lens=lens, max_q_len=S, sinks=sinks)]
        pairs = sum(min(i + 1, s.window or S) for i in range(S))
        return _result(f"{kind}-attn-prefill" + ("-large-scores" if qscale > 1 else ""), args, timer, fns,
                       (2 * q.numel() + k.numel() + v.numel()) * 2, 4.0 * B * H * pairs * V, batch=B, seq=S, window=s.window, heads=H,
                       kv_heads=G, dim=V)
    return case


def attn_decode(kind):
    def case(args, timer, sets_for):
        B, ctx = 64, 1056
        s, sinks = _attn_spec(kind)
        pages, seen = (ctx + 31) // 32, min(s.window or ctx, ctx) + s.keep_first
        nb = B * pages
        sets = sets_for(B * seen * G * 2 * V * 2, args.sets)
        caches = [(_bf16(nb, G, 32, V), _bf16(nb, G, 32, V)) for _ in range(sets)]
        table, lens = _i32(range(nb)).reshape(B, pages), torch.full((B,), ctx, device="cuda", dtype=torch.int32)
        q = _bf16(B, H, V)
        fns = [lambda k=k, v=v: heads_attention(s, q, k, v, table, lens, num_splits=args.kv_splits, sinks=sinks) for k, v in caches]
        return _result(f"{kind}-attn-decode", args, timer, fns, B * seen * G * 2 * V * 2, 4.0 * B * H * seen * V, batch=B, context=ctx,
                       window=s.window, heads=H, kv_heads=G, dim=V, sets=sets)
    return case


def residual(kind, tokens, splits, past=8):
    """tanh: one branch through a norm; average: the same and a weighted sum with `past` earlier results; blend: two normed
    branches through a norm."""
    def case(args, timer, sets_for):
        T = tokens
        part = lambda: Proj(torch.randn(splits, T, W, device="cuda") if splits else _bf16(T, W), 0, W)
        x, w, b = torch.randn(T, W, device="cuda"), _vec(W, 1.0), _vec(W, 0.0)
        norm = Norm(w, b, alpha=0.7)
        br = [Branch(part())] if kind != "blend" else [Branch(part(), norm=w, scale=0.5, shift=b), Branch(part(), norm=w, scale=0.5)]
        hist = History(torch.randn(past + 1, T, W, device="cuda"), past, _vec(past + 1)) if kind == "average" else None
        fns = [lambda: gated_residual(x, br, post=norm, norms=[norm], history=hist, eps=1e-5)]
        per = len(br) * (4 * splits if splits else 2) + 10 + (4 * (past + 1) if hist else 0)
        return _result(f"{kind}-residual-{T}", args, timer, fns, T * W * per, 0.0, tokens=T, width=W, splits=splits,
                       past=past if hist else 0)
    return case


def pair_append(tokens, splits):
    def case(args, timer, sets_for):
        T, s = tokens, MapsSpec(H, G, V, V, V ** -0.5)
        nb, n = max(T // 32, 1) + 8, V * (H + 2 * G)
        k, v = _bf16(nb, G, 32, V), _bf16(nb, G, 32, V)
        y = torch.randn(splits, T, n + H, device="cuda") if splits else _bf16(T, n + H)
        table, pos, slots = torch.randn(4096, V, device="cuda"), _i32(range(T)) % 4096, _i32(range(T))
        fns = [lambda: rope_norm_append(s, Proj(y, 0, H * V), Proj(y, H * V, G * V), Proj(y, (H + G) * V, G * V), None, table, pos,
                                        slots, k, v, norm=False, interleaved=True)]
        return _result(f"pair-append-{T}", args, timer, fns, T * n * ((4 * splits if splits else 2) + 2), 0.0, tokens=T, heads=H,
                       kv_heads=G, dim=V, splits=splits)
    return case


def xielu_gemm(args, timer, sets_for):
    M, N = 8192, 14336
    x, ws = _bf16(M, W), [_bf16(N, W, scale=0.02) for _ in range(2)]
    fns = [lambda w=w: linear(x, w, swap=False, out_act=Act("xielu", 0.8, 0.9)) for w in ws]
    return _result("gemm-prefill-xielu", args, timer, fns, (M * W + N * W + M * N) * 2, 2.0 * M * N * W, M=M, K=W, N=N)


def xielu(args, timer, sets_for):
    T, ff, s = 64, 14336, 4
    y = torch.randn(s, T, ff, device="cuda")
    fns = [lambda: activation(Proj(y, 0, ff), Act("xielu", 0.8, 0.9))]
    return _result("xielu-64", args, timer, fns, T * ff * (4 * s + 2), 0.0, tokens=T, ff=ff, splits=s)


CASES = {"delta-step": rec_step(True), "ssd-step": rec_step(False), "delta-scan": rec_scan(True), "ssd-scan": rec_scan(False),
         "short-conv-16384": conv, "group-norm-64": group_norm(64, 8), "group-norm-16384": group_norm(16384, 0),
         "capped-attn-prefill": attn_prefill("capped"), "capped-attn-prefill-large-scores": attn_prefill("capped", 8.0),
         "capped-attn-decode": attn_decode("capped"), "distance-attn-prefill": attn_prefill("distance"),
         "distance-attn-decode": attn_decode("distance"), "tanh-residual-64": residual("tanh", 64, 8),
         "tanh-residual-16384": residual("tanh", 16384, 0), "average-residual-64": residual("average", 64, 8),
         "average-residual-16384": residual("average", 16384, 0), "blend-residual-64": residual("blend", 64, 8),
         "blend-residual-16384": residual("blend", 16384, 0), "pair-append-64": pair_append(64, 4),
         "pair-append-16384": pair_append(16384, 0), "gemm-prefill-xielu": xielu_gemm, "xielu-64": xielu}
