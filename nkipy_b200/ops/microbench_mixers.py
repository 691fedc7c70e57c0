"""Micro-benchmark cases of the mixed-layer operators (mixers.py), at the shapes of the like kernels of the dense model
(32 query heads, 8 kv heads, 4096 wide, batch 64 or 8 x 2048 tokens)."""
from __future__ import annotations

import torch

from . import grouped_linear, linear, router_topk
from .linear_attention import Decay, linear_attention, linear_state_shape, low_rank, token_mix
from .mixers import (Branch, MapsSpec, Proj, activation, gate_heads, gated_act, gated_residual, heads_attention, hgrn2,
                     hgrn2_state_shape, maps_append, maps_attention, row_norm_append)

H, G, D, V, W = 32, 8, 64, 128, 4096


def _bf16(*shape, scale=1.0):
    return (torch.randn(*shape, device="cuda") * scale).to(torch.bfloat16)


def _i32(x):
    return torch.as_tensor(x, dtype=torch.int32, device="cuda")


def _spec(softcap):
    return MapsSpec(H, G, D, V, D ** -0.5, maps=2, softcap=softcap, lam=0.5, out_scale=0.5, eps=1e-5)


def maps_decode(args, timer, sets_for):
    B, ctx, s = 64, 1056, _spec(30.0)
    pages = (ctx + 31) // 32
    nb = B * pages
    sets = sets_for(nb * G * 32 * (2 * D + V) * 2, args.sets)
    caches = [(_bf16(nb, G, 32, 2 * D), _bf16(nb, G, 32, V)) for _ in range(sets)]
    table, lens = _i32(range(nb)).reshape(B, pages), torch.full((B,), ctx, device="cuda", dtype=torch.int32)
    q = _bf16(B, H, 2 * D)
    fns = [lambda k=k, v=v: maps_attention(s, q, k, v, table, lens, num_splits=args.kv_splits) for k, v in caches]
    return dict(case="maps-attn-decode", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                bytes=B * ctx * G * (2 * D + V) * 2, flops=B * H * ctx * (4.0 * D + 4 * V),
                shape=dict(batch=B, context=ctx, heads=H, kv_heads=G, dim=D, vdim=V, sets=sets))


def maps_prefill(softcap, qscale=1.0, name="maps-attn-prefill"):
    def case(args, timer, sets_for):
        B, S, s = args.batch or 8, args.seq or 2048, _spec(softcap)
        nb = B * S // 32
        k, v, q = _bf16(nb, G, 32, 2 * D), _bf16(nb, G, 32, V), _bf16(B * S, H, 2 * D, scale=qscale)
        table = _i32(range(nb)).reshape(B, S // 32)
        start, lens = _i32(range(B)) * S, torch.full((B,), S, device="cuda", dtype=torch.int32)
        fns = [lambda: maps_attention(s, q, k, v, table, lens, q_start=start, q_lens=lens, max_q_len=S)]
        return dict(case=name, us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=(q.numel() + k.numel() + v.numel() + B * S * H * V) * 2,
                    flops=B * H * S * S / 2 * (4.0 * D + 4 * V),
                    shape=dict(batch=B, seq=S, heads=H, kv_heads=G, dim=D, vdim=V, softcap=softcap, q_scale=qscale))
    return case


def append(args, timer, sets_for):
    B, S, s = args.batch or 8, args.seq or 2048, _spec(30.0)
    T, nb, n = B * S, B * S // 32, 2 * D * (H + G) + V * G
    k, v = _bf16(nb, G, 32, 2 * D), _bf16(nb, G, 32, V)
    y = _bf16(T, n + W)
    table = torch.randn(S, D, device="cuda")
    pos, slots = _i32(range(T)) % S, _i32(range(T))
    c1, c2 = 2 * D * H, 2 * D * (H + G)
    fns = [lambda: maps_append(s, Proj(y, 0, c1), Proj(y, c1, c2 - c1), Proj(y, c2, V * G), table, pos, slots, k, v)]
    return dict(case="maps-append", us=timer(fns, args.iters, args.warmup, not args.no_graph), bytes=2 * T * n * 2, flops=0.0,
                shape=dict(tokens=T, heads=H, kv_heads=G))


def _rec(T, sets):
    y = [_bf16(T, 3 * W + W) for _ in range(sets)]
    sl = lambda t: (Proj(t, 0, W), Proj(t, W, W), Proj(t, 2 * W, W))
    w = [torch.randn(W, device="cuda"), torch.rand(W, device="cuda"), torch.ones(V, device="cuda")]
    return y, sl, w


def rec_step(args, timer, sets_for):
    B = 64
    state_bytes = B * H * V * V * 4
    sets = sets_for(2 * state_bytes, args.sets)
    y, sl, w = _rec(B, 1)
    states = [torch.randn(B, *hgrn2_state_shape(H, V, V), device="cuda") for _ in range(sets)]
    lens = torch.full((B,), 77, device="cuda", dtype=torch.int32)
    fns = [lambda st=st: hgrn2(*sl(y[0]), *w, st, lens, heads=H, dim=V, vdim=V, eps=1e-5) for st in states]
    return dict(case="hgrn2-step", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                bytes=2 * state_bytes + B * W * 8, flops=B * H * V * V * 5.0,
                shape=dict(batch=B, heads=H, dim=V, vdim=V, sets=sets))


def rec_scan(args, timer, sets_for):
    B, S = args.batch or 8, args.seq or 2048
    y, sl, w = _rec(B * S, 1)
    state = torch.zeros(B, *hgrn2_state_shape(H, V, V), device="cuda")
    start, lens = _i32(range(B)) * S, torch.full((B,), S, device="cuda", dtype=torch.int32)
    rows = _i32(range(B))
    fns = [lambda: hgrn2(*sl(y[0]), *w, state, lens, heads=H, dim=V, vdim=V, eps=1e-5, q_start=start, q_lens=lens,
                         rows=rows)]
    # bytes: q, f, v in, o out and through the head norm once more
    return dict(case="hgrn2-scan", us=timer(fns, args.iters, args.warmup, not args.no_graph), bytes=B * S * W * 2 * 6,
                flops=B * S * H * V * V * 5.0, shape=dict(batch=B, seq=S, heads=H, dim=V, vdim=V))


def residual(tokens, splits):
    def case(args, timer, sets_for):
        T = tokens
        mk = (lambda: torch.randn(splits, T, W, device="cuda")) if splits else (lambda: _bf16(T, W))
        x, y1, g1, y2, g2 = torch.randn(T, W, device="cuda"), mk(), mk(), mk(), mk()
        b, n = torch.randn(W, device="cuda"), torch.ones(W, device="cuda")
        br = [(Proj(y1, 0, W), Proj(g1, 0, W), b), (Proj(y2, 0, W), Proj(g2, 0, W), b)]
        fns = [lambda: gated_residual(x, br, norms=[n, n], groups=4, eps=1e-5)]
        per = 4 * (4 * splits if splits else 2) + 8 + 4
        return dict(case=f"gated-residual-{tokens}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * W * per, flops=0.0, shape=dict(tokens=T, width=W, splits=splits))
    return case


def act(args, timer, sets_for):
    T, ff, s = 64, 14336, 1
    y = torch.randn(s, T, 2 * ff, device="cuda")
    fns = [lambda: gated_act(Proj(y, 0, ff), Proj(y, ff, ff), "gelu_tanh")]
    return dict(case="gated-act-64", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                bytes=T * ff * (8 * s + 2), flops=0.0, shape=dict(tokens=T, ff=ff, splits=s))


# --------------------------------------------------------------------------- linear attention and its surroundings
R = 64                       # width of the low-rank projections


def _lin(T, kind, seed_rows=1):
    """(projection slices q, k, v, gate, low-rank input), decay and keyword arguments of 32 heads of 128 x 128."""
    y = _bf16(T, 4 * W + R)
    q, k, v, g = (Proj(y, i * W, W) for i in range(4))
    bias = torch.randn(W, device="cuda") + (1.0 if kind == "gla" else -4.0)
    decay = Decay("sigmoid_root" if kind == "gla" else "double_exp", Proj(y, 4 * W, R), _bf16(W, R, scale=0.1), bias,
                  "none" if kind == "gla" else "tanh", 16.0)
    norm = torch.ones(V if kind == "gla" else W, device="cuda")
    kw = dict(heads=H, dim=V, vdim=V, eps=1e-6, bonus=None if kind == "gla" else torch.randn(W, device="cuda"))
    return (q, k, v, decay, g, norm), kw


def lin_step(kind):
    def case(args, timer, sets_for):
        B = 64
        state_bytes = B * H * V * V * 4
        sets = sets_for(2 * state_bytes, args.sets)
        a, kw = _lin(B, kind)
        states = [torch.randn(B, *linear_state_shape(H, V, V), device="cuda") for _ in range(sets)]
        lens = torch.full((B,), 77, device="cuda", dtype=torch.int32)
        fns = [lambda st=st: linear_attention(*a, st, lens, **kw) for st in states]
        return dict(case=f"{kind}-step", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=2 * state_bytes + B * W * 10, flops=B * H * V * V * 5.0,
                    shape=dict(batch=B, heads=H, dim=V, vdim=V, rank=R, sets=sets))
    return case


def lin_scan(kind):
    def case(args, timer, sets_for):
        B, S = args.batch or 8, args.seq or 2048
        a, kw = _lin(B * S, kind)
        state = torch.zeros(B, *linear_state_shape(H, V, V), device="cuda")
        start, lens = _i32(range(B)) * S, torch.full((B,), S, device="cuda", dtype=torch.int32)
        fns = [lambda: linear_attention(*a, state, lens, q_start=start, q_lens=lens, rows=_rows, **kw)]
        _rows = _i32(range(B))
        # bytes: q, k, v, gate in, o out and through the head norm once more, logits of the decay in fp32 out and in
        return dict(case=f"{kind}-scan", us=timer(fns, args.iters, args.warmup, not args.no_graph), bytes=B * S * W * (2 * 7 + 8),
                    flops=B * S * H * V * V * 5.0, shape=dict(batch=B, seq=S, heads=H, dim=V, vdim=V, rank=R))
    return case


def mix(tokens):
    def case(args, timer, sets_for):
        T = tokens
        B = 64 if T <= 64 else 8
        h, mu, st = _bf16(T, W), torch.rand(5, W, device="cuda"), torch.zeros(B, W, device="cuda")
        n = T // B
        lens = torch.full((B,), n + (n == 1), device="cuda", dtype=torch.int32)
        kw = {} if n == 1 else dict(q_start=_i32(range(B)) * n, q_lens=lens)
        fns = [lambda: token_mix(h, mu, st, lens, **kw)]
        return dict(case=f"token-mix-{T}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * W * 12 + (B * W * 8 if n == 1 else 0), flops=0.0, shape=dict(tokens=T, width=W, mixes=5))
    return case


def row_append(tokens, splits):
    def case(args, timer, sets_for):
        T, s = tokens, MapsSpec(H, G, V, V, V ** -0.5, maps=1, window=1024)
        nb, n = max(T // 32, 1) + 8, V * (H + 2 * G)
        k, v = _bf16(nb, G, 32, V), _bf16(nb, G, 32, V)
        y = torch.randn(splits, T, n + W, device="cuda") if splits else _bf16(T, n + W)
        slots = _i32(range(T))
        qn, kn = torch.ones(H * V, device="cuda"), torch.ones(G * V, device="cuda")
        fns = [lambda: row_norm_append(s, Proj(y, 0, H * V), Proj(y, H * V, G * V), Proj(y, (H + G) * V, G * V), qn, kn, slots,
                                       k, v)]
        return dict(case=f"row-norm-append-{T}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * n * ((4 * splits if splits else 2) + 2), flops=0.0,
                    shape=dict(tokens=T, heads=H, kv_heads=G, dim=V, splits=splits))
    return case


def gates(tokens):
    def case(args, timer, sets_for):
        T = tokens
        x, g = _bf16(T, H, V), _bf16(T, W)
        out = _bf16(T, 2 * W)
        fns = [lambda: gate_heads(x, Proj(g, 0, W), "sigmoid", scale=0.7, out=out[:, :W])]
        return dict(case=f"gate-heads-{T}", us=timer(fns, args.iters, args.warmup, not args.no_graph), bytes=T * W * 6,
                    flops=0.0, shape=dict(tokens=T, heads=H, width=V))
    return case


def window_decode(window):
    def case(args, timer, sets_for):
        B, ctx, s = 64, 1056, MapsSpec(H, G, V, V, V ** -0.5, maps=1, window=window)
        pages = (ctx + 31) // 32
        nb, seen = B * pages, min(window or ctx, ctx)
        sets = sets_for(B * seen * G * 2 * V * 2, args.sets)
        caches = [(_bf16(nb, G, 32, V), _bf16(nb, G, 32, V)) for _ in range(sets)]
        table, lens = _i32(range(nb)).reshape(B, pages), torch.full((B,), ctx, device="cuda", dtype=torch.int32)
        q = _bf16(B, H, V)
        fns = [lambda k=k, v=v: heads_attention(s, q, k, v, table, lens, num_splits=args.kv_splits) for k, v in caches]
        return dict(case="window-attn-decode", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=B * seen * G * 2 * V * 2, flops=4.0 * B * H * seen * V,
                    shape=dict(batch=B, context=ctx, window=window, heads=H, kv_heads=G, dim=V, sets=sets))
    return case


def window_prefill(window):
    def case(args, timer, sets_for):
        B, S, s = args.batch or 8, args.seq or 2048, MapsSpec(H, G, V, V, V ** -0.5, maps=1, window=window)
        nb = B * S // 32
        k, v, q = _bf16(nb, G, 32, V), _bf16(nb, G, 32, V), _bf16(B * S, H, V)
        table = _i32(range(nb)).reshape(B, S // 32)
        start, lens = _i32(range(B)) * S, torch.full((B,), S, device="cuda", dtype=torch.int32)
        fns = [lambda: heads_attention(s, q, k, v, table, lens, q_start=start, q_lens=lens, max_q_len=S)]
        pairs = sum(min(i + 1, window) for i in range(S))
        return dict(case="window-attn-prefill", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=(2 * q.numel() + k.numel() + v.numel()) * 2, flops=4.0 * B * H * pairs * V,
                    shape=dict(batch=B, seq=S, window=window, heads=H, kv_heads=G, dim=V))
    return case


def each(args, timer, sets_for):
    T = 64
    sets = sets_for(4 * W * W * 2, args.sets)
    ws, x = [_bf16(4, W, W, scale=0.02) for _ in range(sets)], _bf16(4 * T, W)
    off = _i32(range(5)) * T
    fns = [lambda w=w: grouped_linear(x, w, off, max_rows_per_group=T) for w in ws]
    return dict(case="grouped-projections-64", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                bytes=4 * W * W * 2 + 8 * T * W * 2, flops=8.0 * T * W * W, shape=dict(tokens=T, groups=4, k=W, n=W, sets=sets))


def plain_residual(tokens, splits):
    def case(args, timer, sets_for):
        T = tokens
        y = torch.randn(splits, T, W, device="cuda") if splits else _bf16(T, W)
        x, n = torch.randn(T, W, device="cuda"), torch.ones(W, device="cuda")
        fns = [lambda: gated_residual(x, [Branch(Proj(y, 0, W))], norms=[n], eps=1e-6)]
        return dict(case=f"residual-{tokens}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * W * ((4 * splits if splits else 2) + 10), flops=0.0, shape=dict(tokens=T, width=W, splits=splits))
    return case


def routed_residual(tokens):
    def case(args, timer, sets_for):
        T, k = tokens, 4
        y, x, n = _bf16(T * k, W), torch.randn(T, W, device="cuda"), torch.ones(W, device="cuda")
        pos, pw = torch.randperm(T * k, device="cuda").to(torch.int32), torch.rand(T, k, device="cuda")
        fns = [lambda: gated_residual(x, [Branch(Proj(y, 0, W), pair_pos=pos, pair_w=pw)], norms=[n], eps=1e-6)]
        return dict(case=f"routed-residual-{tokens}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * W * (2 * k + 10), flops=0.0, shape=dict(tokens=T, width=W, top=k))
    return case


def router(tokens):
    def case(args, timer, sets_for):
        T, E = tokens, 128
        z = torch.randn(8, T, E, device="cuda")
        fns = [lambda: router_topk(z, 8, groups=8, keep=4, scale=2.0)]
        return dict(case=f"group-router-{T}", us=timer(fns, args.iters, args.warmup, not args.no_graph), bytes=z.numel() * 4,
                    flops=0.0, shape=dict(tokens=T, experts=E, top=8, groups=8, keep=4, splits=8))
    return case


def decay_logits(tokens):
    def case(args, timer, sets_for):
        x, w = _bf16(tokens, R), _bf16(W, R)
        fns = [lambda: low_rank(Proj(x, 0, R), w, "tanh")]
        return dict(case=f"low-rank-{tokens}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=tokens * W * 4 + W * R * 2, flops=2.0 * tokens * W * R, shape=dict(tokens=tokens, rank=R, width=W))
    return case


def relu2_gemm(args, timer, sets_for):
    M, N = 8192, 14336
    x, ws = _bf16(M, W), [_bf16(N, W, scale=0.02) for _ in range(2)]
    fns = [lambda w=w: linear(x, w, swap=False, out_act="relu2") for w in ws]
    return dict(case="gemm-prefill-relu2", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                bytes=(M * W + N * W + M * N) * 2, flops=2.0 * M * N * W, shape=dict(M=M, K=W, N=N))


def relu2(args, timer, sets_for):
    T, ff, s = 64, 14336, 4
    y = torch.randn(s, T, ff, device="cuda")
    fns = [lambda: activation(Proj(y, 0, ff), "relu2")]
    return dict(case="relu2-64", us=timer(fns, args.iters, args.warmup, not args.no_graph), bytes=T * ff * (4 * s + 2), flops=0.0,
                shape=dict(tokens=T, ff=ff, splits=s))


CASES = {"maps-attn-decode": maps_decode, "maps-attn-prefill": maps_prefill(30.0),
         "maps-attn-prefill-large-scores": maps_prefill(30.0, 8.0, "maps-attn-prefill-large-scores"),
         "maps-attn-prefill-nocap": maps_prefill(0.0, 1.0, "maps-attn-prefill-nocap"), "maps-append": append,
         "hgrn2-step": rec_step, "hgrn2-scan": rec_scan, "gated-residual-64": residual(64, 8),
         "gated-residual-16384": residual(16384, 0), "gated-act-64": act,
         "gla-step": lin_step("gla"), "rwkv-step": lin_step("rwkv"), "gla-scan": lin_scan("gla"), "rwkv-scan": lin_scan("rwkv"),
         "token-mix-64": mix(64), "token-mix-16384": mix(16384), "row-norm-append-64": row_append(64, 4),
         "row-norm-append-16384": row_append(16384, 0), "gate-heads-64": gates(64), "gate-heads-16384": gates(16384),
         "window-attn-decode": window_decode(1024), "window-attn-prefill": window_prefill(1024),
         "grouped-projections-64": each, "residual-64": plain_residual(64, 8), "residual-16384": plain_residual(16384, 0),
         "routed-residual-64": routed_residual(64), "routed-residual-16384": routed_residual(16384),
         "group-router-64": router(64), "group-router-16384": router(16384), "low-rank-64": decay_logits(64),
         "low-rank-16384": decay_logits(16384), "gemm-prefill-relu2": relu2_gemm, "relu2-64": relu2}
