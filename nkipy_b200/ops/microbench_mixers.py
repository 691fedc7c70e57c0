"""Micro-benchmark cases of the mixed-layer operators (mixers.py), at the shapes of the like kernels of the dense model
(32 query heads, 8 kv heads, 4096 wide, batch 64 or 8 x 2048 tokens)."""
from __future__ import annotations

import torch

from . import grouped_linear, head_linear, linear, moe_dispatch, router_topk, softcap
from .latent_attention import (LatentSpec, latent_append, latent_attention, latent_gather, latent_prefill, latent_queries)
from .linear_attention import Decay, linear_attention, linear_state_shape, low_rank, token_mix
from .mixers import (Branch, MapsSpec, Norm, Proj, activation, gate_heads, gated_act, gated_residual, heads_attention, hgrn2,
                     hgrn2_state_shape, maps_append, maps_attention, row_norm_append, rope_norm_append)

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


# latent attention: heads of 128 unrotated and 64 rotated dimensions, latents of 512 (keys, values) and 1536 (queries)
LAT = dict(dim=128, rot=64, vdim=V, rank=512, q_rank=1536, scale=192 ** -0.5)


def latent_decode(heads, window):
    def case(args, timer, sets_for):
        B, ctx, s = 64, 1056, LatentSpec(heads, window=window, **LAT)
        pages, seen = (ctx + 31) // 32, min(window or ctx, ctx)
        nb = B * pages
        sets = sets_for(B * seen * s.row * 2, args.sets)
        caches = [_bf16(nb, 1, 32, s.row) for _ in range(sets)]
        table, lens = _i32(range(nb)).reshape(B, pages), torch.full((B,), ctx, device="cuda", dtype=torch.int32)
        q, sinks = _bf16(heads, B, s.row), torch.zeros(heads, device="cuda")
        fns = [lambda c=c: latent_attention(s, q, c, table, lens, sinks=sinks, num_splits=args.kv_splits) for c in caches]
        return dict(case=f"latent-attn-decode-{heads}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=B * seen * s.row * 2 + B * heads * (s.row + s.rank) * 2,
                    flops=2.0 * B * heads * seen * (s.rank + s.rot + s.rank),
                    shape=dict(batch=B, context=ctx, window=window, heads=heads, rank=s.rank, rot=s.rot, sets=sets))
    return case


def latent_pf(dim, window):
    def case(args, timer, sets_for):
        B, S, s = args.batch or 8, args.seq or 2048, LatentSpec(H, window=window, **{**LAT, "dim": dim})
        T, nk = B * S, s.slabs[0]
        q, kv, r = _bf16(T, H, 64 * nk), _bf16(T, H * (s.dim + s.vdim)), _bf16(T, s.rot)
        start, lens, sinks = _i32(range(B)) * S, torch.full((B,), S, device="cuda", dtype=torch.int32), torch.zeros(H, device="cuda")
        fns = [lambda: latent_prefill(s, q, kv, r, start, start, lens, lens, S, sinks)]
        pairs = sum(min(i + 1, window or S) for i in range(S))
        return dict(case=f"latent-attn-prefill-{dim}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=(q.numel() + kv.numel() + r.numel() + T * H * V) * 2, flops=2.0 * B * H * pairs * (s.dim + s.rot + s.vdim),
                    shape=dict(batch=B, seq=S, window=window, heads=H, dim=s.dim, rot=s.rot, vdim=s.vdim))
    return case


def chunk_pf(chunk):
    def case(args, timer, sets_for):
        B, S, s = args.batch or 8, args.seq or 2048, MapsSpec(H, G, V, V, V ** -0.5, maps=1, chunk=chunk)
        nb = B * S // 32
        k, v, q = _bf16(nb, G, 32, V), _bf16(nb, G, 32, V), _bf16(B * S, H, V)
        table = _i32(range(nb)).reshape(B, S // 32)
        start, lens = _i32(range(B)) * S, torch.full((B,), S, device="cuda", dtype=torch.int32)
        fns = [lambda: heads_attention(s, q, k, v, table, lens, q_start=start, q_lens=lens, max_q_len=S)]
        pairs = sum(i % chunk + 1 for i in range(S))
        return dict(case="chunk-attn-prefill", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=(2 * q.numel() + k.numel() + v.numel()) * 2, flops=4.0 * B * H * pairs * V,
                    shape=dict(batch=B, seq=S, chunk=chunk, heads=H, kv_heads=G, dim=V))
    return case


def chunk_decode(chunk):
    def case(args, timer, sets_for):
        B, ctx, s = 64, 2 * chunk, MapsSpec(H, G, V, V, V ** -0.5, maps=1, chunk=chunk)
        pages = ctx // 32
        nb = B * pages
        sets = sets_for(B * chunk * G * 2 * V * 2, min(args.sets, 3))
        caches = [(_bf16(nb, G, 32, V), _bf16(nb, G, 32, V)) for _ in range(sets)]
        table, lens = _i32(range(nb)).reshape(B, pages), torch.full((B,), ctx, device="cuda", dtype=torch.int32)
        q = _bf16(B, H, V)
        fns = [lambda k=k, v=v: heads_attention(s, q, k, v, table, lens, num_splits=args.kv_splits) for k, v in caches]
        return dict(case="chunk-attn-decode", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=B * chunk * G * 2 * V * 2, flops=4.0 * B * H * chunk * V,
                    shape=dict(batch=B, context=ctx, chunk=chunk, heads=H, kv_heads=G, dim=V, sets=sets))
    return case


def latent_app(tokens, splits):
    def case(args, timer, sets_for):
        T, s = tokens, LatentSpec(H, window=1024, **LAT)
        n = s.q_rank + s.rank + s.rot
        y = torch.randn(splits, T, n + H, device="cuda") if splits else _bf16(T, n + H)
        cache, slots = _bf16(max(T // 32, 1) + 8, 1, 32, s.row), _i32(range(T))
        table, pos = torch.randn(4096, s.rot, device="cuda"), _i32(range(T)) % 4096
        qn, kn = torch.ones(s.q_rank, device="cuda"), torch.ones(s.rank, device="cuda")
        fns = [lambda: latent_append(s, Proj(y, 0, s.q_rank), Proj(y, s.q_rank, s.rank + s.rot), qn, kn, table, pos, slots, cache)]
        return dict(case=f"latent-append-{T}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * n * ((4 * splits if splits else 2) + 2), flops=0.0,
                    shape=dict(tokens=T, q_rank=s.q_rank, rank=s.rank, rot=s.rot, splits=splits))
    return case


def latent_q(tokens, splits):
    def case(args, timer, sets_for):
        T, s = tokens, LatentSpec(H, window=1024, **LAT)
        n = H * (s.dim + s.rot)
        y = torch.randn(splits, T, n, device="cuda") if splits else _bf16(T, n)
        table, pos = torch.randn(4096, s.rot, device="cuda"), _i32(range(T)) % 4096
        if splits:
            q = _bf16(H, T, s.row)
            plain, rot = _bf16(H, T, s.dim).transpose(0, 1), q.transpose(0, 1)[..., s.rank:]
        else:
            q = _bf16(T, H, 64 * s.slabs[0])
            plain, rot = q[..., :-64], q[..., -64:]
        fns = [lambda: latent_queries(s, Proj(y, 0, n), table, pos, plain, rot)]
        return dict(case=f"latent-queries-{T}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * n * ((4 * splits if splits else 2) + 2), flops=0.0,
                    shape=dict(tokens=T, heads=H, dim=s.dim, rot=s.rot, splits=splits))
    return case


def latent_rows(args, timer, sets_for):
    P, s = 512, LatentSpec(H, window=1024, **LAT)
    cache = _bf16(2 * P, 1, 32, s.row)
    pages = torch.randperm(2 * P, device="cuda").to(torch.int32)[:P].contiguous()
    fns = [lambda: latent_gather(s, cache, pages, s.rot)]
    return dict(case="latent-gather-16384", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                bytes=4 * P * 32 * (s.rank + s.rot), flops=0.0, shape=dict(pages=P, rank=s.rank, rot=s.rot))


def fold(k, n, name):
    def case(args, timer, sets_for):
        T = 64
        sets = sets_for(H * n * k * 2, 32)
        ws, x = [_bf16(H, n, k, scale=0.05) for _ in range(sets)], _bf16(H, T, k)
        fns = [lambda w=w: head_linear(x, w) for w in ws]
        return dict(case=name, us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=H * (n * k + T * (n + k)) * 2, flops=2.0 * H * T * n * k, shape=dict(tokens=T, heads=H, k=k, n=n, sets=sets))
    return case


def rope_append(tokens, splits):
    def case(args, timer, sets_for):
        T, s = tokens, MapsSpec(H, G, V, V, V ** -0.5, maps=1, chunk=1024)
        nb, n = max(T // 32, 1) + 8, V * (H + 2 * G)
        k, v = _bf16(nb, G, 32, V), _bf16(nb, G, 32, V)
        y = torch.randn(splits, T, n + H, device="cuda") if splits else _bf16(T, n + H)
        slots, bias = _i32(range(T)), torch.randn(n, device="cuda")
        table, pos = torch.randn(4096, V, device="cuda"), _i32(range(T)) % 4096
        fns = [lambda: rope_norm_append(s, Proj(y, 0, H * V), Proj(y, H * V, G * V), Proj(y, (H + G) * V, G * V), bias, table, pos,
                                        slots, k, v)]
        return dict(case=f"rope-norm-append-{T}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * n * ((4 * splits if splits else 2) + 2), flops=0.0,
                    shape=dict(tokens=T, heads=H, kv_heads=G, dim=V, splits=splits))
    return case


def head_gates(tokens):
    def case(args, timer, sets_for):
        T = tokens
        x, g = _bf16(T, H, V), _bf16(T, H)
        fns = [lambda: gate_heads(x, Proj(g, 0, H), "sigmoid")]
        return dict(case=f"head-gates-{T}", us=timer(fns, args.iters, args.warmup, not args.no_graph), bytes=T * W * 4,
                    flops=0.0, shape=dict(tokens=T, heads=H, width=V))
    return case


def side_residual(tokens, splits):
    def case(args, timer, sets_for):
        T = tokens
        y = torch.randn(splits, T, W, device="cuda") if splits else _bf16(T, W)
        x, n, b = torch.randn(T, W, device="cuda"), torch.ones(W, device="cuda"), torch.zeros(W, device="cuda")
        fns = [lambda: gated_residual(x, [Branch(Proj(y, 0, W), norm=n)], norms=[Norm(n, b, True)], eps=1e-6)]
        return dict(case=f"normed-residual-{tokens}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * W * ((4 * splits if splits else 2) + 10), flops=0.0, shape=dict(tokens=T, width=W, splits=splits))
    return case


def parallel_residual(tokens, splits, routed):
    def case(args, timer, sets_for):
        T, k = tokens, 4
        part = lambda: torch.randn(splits, T, W, device="cuda") if splits else _bf16(T, W)
        x, br = torch.randn(T, W, device="cuda"), [Branch(Proj(part(), 0, W))]
        per = 4 * splits if splits else 2
        size = per
        if routed:
            rows, pos = _bf16(T * k, W), torch.randperm(T * k, device="cuda").to(torch.int32)
            gate = torch.randn(2, T, 40, device="cuda")
            br += [Branch(Proj(rows, 0, W), pair_pos=pos, top_k=k), Branch(Proj(part(), 0, W), Proj(gate, 32, 1))]
            size += 2 * k + per
        else:
            br.append(Branch(Proj(part(), 0, W)))
            size += per
        fns = [lambda: gated_residual(x, br, norms=[Norm()])]
        name = "shared-routed-residual" if routed else "parallel-residual"
        return dict(case=f"{name}-{tokens}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * W * (size + 10), flops=0.0, shape=dict(tokens=T, width=W, splits=splits, top=k if routed else 0))
    return case


def table_act(tokens, splits):
    def case(args, timer, sets_for):
        T, n, L, vocab = tokens, 256, 16, 32000
        z = torch.randn(splits, T, n, device="cuda") if splits else _bf16(T, n)
        table, ids = _bf16(vocab, L * n), torch.randint(0, vocab, (T,), device="cuda", dtype=torch.int32)
        fns = [lambda i=i: gated_act(Proj(z, 0, n), Proj(table, i * n, n), "gelu_tanh", up_rows=ids) for i in range(4)]
        return dict(case=f"table-act-{T}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * n * ((4 * splits if splits else 2) + 4), flops=0.0, shape=dict(tokens=T, width=n, splits=splits))
    return case


def clamped_act(tokens, splits):
    def case(args, timer, sets_for):
        T, ff = tokens, 1792
        y = torch.randn(splits, T, 2 * ff, device="cuda") if splits else _bf16(T, 2 * ff)
        fns = [lambda: gated_act(Proj(y, 0, ff), Proj(y, ff, ff), "clamped", limit=7.0)]
        return dict(case=f"clamped-act-{T}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * ff * (2 * (4 * splits if splits else 2) + 2), flops=0.0, shape=dict(tokens=T, ff=ff, splits=splits))
    return case


def sigmoid_router(tokens, splits):
    def case(args, timer, sets_for):
        T, E = tokens, 32
        z = torch.randn(splits, T, E + 8, device="cuda")
        fns = [lambda: router_topk(Proj(z, 0, E), 4, "sigmoid_topk")]
        return dict(case=f"sigmoid-router-{T}", us=timer(fns, args.iters, args.warmup, not args.no_graph), bytes=splits * T * E * 4,
                    flops=0.0, shape=dict(tokens=T, experts=E, top=4, splits=splits))
    return case


def scaled_dispatch(tokens, scaled):
    def case(args, timer, sets_for):
        T, k, E = tokens, 4, 32
        x, e = _bf16(T, W), torch.rand(T, E, device="cuda").topk(k, dim=-1).indices.to(torch.int32)
        w = torch.rand(T, k, device="cuda") if scaled else None
        fns = [lambda: moe_dispatch(x, e, 0, E, weights=w)]
        return dict(case=f"{'scaled' if scaled else 'plain'}-dispatch-{T}", us=timer(fns, args.iters, args.warmup, not args.no_graph),
                    bytes=T * W * 2 * (k + 1), flops=0.0, shape=dict(tokens=T, width=W, experts=E, top=k))
    return case


def cap(args, timer, sets_for):
    z = torch.randn(64, 32000, device="cuda")
    fns = [lambda: softcap(z, 30.0)]
    return dict(case="softcap-64", us=timer(fns, args.iters, args.warmup, not args.no_graph), bytes=z.numel() * 8, flops=0.0,
                shape=dict(rows=64, vocab=32000))


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
         "low-rank-16384": decay_logits(16384), "gemm-prefill-relu2": relu2_gemm, "relu2-64": relu2,
         "latent-attn-decode-32": latent_decode(32, 1024), "latent-attn-decode-16": latent_decode(16, 1024),
         "latent-attn-prefill-128": latent_pf(128, 1024), "latent-attn-prefill-64": latent_pf(64, 1024),
         "chunk-attn-prefill": chunk_pf(1024), "chunk-attn-decode": chunk_decode(1024),
         "latent-append-64": latent_app(64, 4), "latent-append-16384": latent_app(16384, 0), "latent-queries-64": latent_q(64, 4),
         "latent-queries-16384": latent_q(16384, 0), "latent-gather-16384": latent_rows,
         "fold-queries-64": fold(128, 512, "fold-queries-64"), "expand-values-64": fold(512, 128, "expand-values-64"),
         "rope-norm-append-64": rope_append(64, 4), "rope-norm-append-16384": rope_append(16384, 0),
         "head-gates-64": head_gates(64), "head-gates-16384": head_gates(16384), "normed-residual-64": side_residual(64, 4),
         "normed-residual-16384": side_residual(16384, 0), "parallel-residual-64": parallel_residual(64, 8, False),
         "parallel-residual-16384": parallel_residual(16384, 0, False),
         "shared-routed-residual-64": parallel_residual(64, 8, True),
         "shared-routed-residual-16384": parallel_residual(16384, 0, True), "table-act-64": table_act(64, 8),
         "table-act-16384": table_act(16384, 0), "clamped-act-64": clamped_act(64, 4),
         "clamped-act-16384": clamped_act(16384, 0), "sigmoid-router-64": sigmoid_router(64, 4),
         "sigmoid-router-16384": sigmoid_router(16384, 2), "scaled-dispatch-64": scaled_dispatch(64, True),
         "scaled-dispatch-16384": scaled_dispatch(16384, True), "plain-dispatch-64": scaled_dispatch(64, False),
         "plain-dispatch-16384": scaled_dispatch(16384, False), "softcap-64": cap}
