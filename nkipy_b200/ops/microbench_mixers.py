"""Micro-benchmark cases of the mixed-layer operators (mixers.py), at the shapes of the like kernels of the dense model
(32 query heads, 8 kv heads, 4096 wide, batch 64 or 8 x 2048 tokens)."""
from __future__ import annotations

import torch

from .mixers import MapsSpec, Proj, gated_act, gated_residual, hgrn2, hgrn2_state_shape, maps_append, maps_attention

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


CASES = {"maps-attn-decode": maps_decode, "maps-attn-prefill": maps_prefill(30.0),
         "maps-attn-prefill-large-scores": maps_prefill(30.0, 8.0, "maps-attn-prefill-large-scores"),
         "maps-attn-prefill-nocap": maps_prefill(0.0, 1.0, "maps-attn-prefill-nocap"), "maps-append": append,
         "hgrn2-step": rec_step, "hgrn2-scan": rec_scan, "gated-residual-64": residual(64, 8),
         "gated-residual-16384": residual(16384, 0), "gated-act-64": act}
