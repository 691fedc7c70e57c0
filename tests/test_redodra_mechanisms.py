"""Each mechanism of the sandwich layer-by-layer decoders against the plain statement in redodra_oracle.py: the operators' PyTorch
form on the CPU and the kernels on a GPU, in 32-bit and in bfloat16."""
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import redodra_oracle as O  # noqa: E402

from nkipy_b200 import ops  # noqa: E402
from nkipy_b200.ops import Act, Branch, HeadRecurrence, MapsSpec, Norm, Proj, ShortConv  # noqa: E402
from nkipy_b200.ops.mixers import History, _post_residual  # noqa: E402

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
on_devices = pytest.mark.parametrize("device", DEVICES)
in_dtypes = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}


@pytest.fixture(autouse=True, scope="module")
def _one_thread():
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def rnd(*shape, seed=0, std=1.0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * std


def close(got, want, tol, what=""):
    got, want = got.double().cpu(), want.double()
    err = ((got - want).abs().max() / want.abs().max().clamp(min=1e-6)).item()
    assert err < tol, f"{what} relative error {err}"


def near(got, want, dtype, what=""):
    """Worst error in 32-bit; in bfloat16, where a norm can blow up the rounding of a small row, the error of the whole."""
    if dtype == torch.float32:
        return close(got, want, 1e-4, what)
    err = ((got.double() - want).norm() / want.norm()).item()
    assert err < 1.2e-2, f"{what} relative error {err}"


def projection(x, form):
    """x fp32 [T, N] as finished values ("f32", "bf16") or as three partial sums, and the values it stands for."""
    if form == "bf16":
        return x.bfloat16(), x.bfloat16().double()
    if form == "partials":
        a, b = rnd(*x.shape, seed=5), rnd(*x.shape, seed=6)
        return torch.stack([a, b, x - a - b]), (a.double() + b.double() + (x - a - b).double())
    return x, x.double()


def form_of(dtype, tokens):
    return "f32" if dtype == torch.float32 else ("bf16" if tokens > 8 else "partials")


def i32(x, device):
    return torch.tensor(x, dtype=torch.int32, device=device)


# --------------------------------------------------------------------------- residual, norms
def tanh_norm(width, seed, device, alpha=0.7):
    w, b = 1 + rnd(width, seed=seed), rnd(width, seed=seed + 1)
    return Norm(w.to(device), b.to(device), alpha=alpha), lambda x: O.tanh_norm(x, alpha, w.double(), b.double())


@on_devices
@in_dtypes
@pytest.mark.parametrize("form", ["f32", "bf16", "partials"])
@pytest.mark.parametrize("width", [96, 70, 2052])
@pytest.mark.parametrize("size", [1e-2, 1.0, 40.0])
def test_tanh_norms_before_and_after(device, dtype, form, width, size):
    """Small arguments (where tanh is its argument), middle ones and saturated ones."""
    T = 5
    x = rnd(T, width, seed=1, std=size)
    y, yv = projection(rnd(T, width + 4, seed=4, std=size), "f32" if form == "partials" and size < 1 else form)
    (post, f), (n1, g1), (n2, g2) = (tanh_norm(width, s, device, a) for s, a in ((10, 1.3), (20, 0.4), (30, 2.0)))
    r, (h1, h2) = ops.gated_residual(x.to(device), [Branch(Proj(y.to(device), 4, width))], post=post, norms=[n1, n2], dtype=dtype)
    want = x.double() + f(yv[:, 4:])
    close(r, want, TOL[torch.float32] if dtype == torch.float32 else 1e-4, "residual")
    close(h1, g1(want), TOL[dtype], "norm")
    close(h2, g2(want), TOL[dtype], "second norm")


@on_devices
@in_dtypes
@pytest.mark.parametrize("form", ["f32", "bf16", "partials"])
@pytest.mark.parametrize("width", [96, 70, 2048, 9000])
def test_mean_of_two_normed_branches_through_a_norm(device, dtype, form, width):
    T, eps = 4, 1e-3
    x, wa, wb, shift = rnd(T, width, seed=1), 1 + rnd(width, seed=2), 1 + rnd(width, seed=3), rnd(width, seed=4)
    scale = torch.tensor([1e-2, 0.1, 1.0, 30.0])[:, None]
    a, av = projection(rnd(T, width, seed=5) * scale, "f32" if form == "partials" else form)
    b, bv = projection(rnd(T, width, seed=6), form)
    (post, f), (norm, g) = tanh_norm(width, 10, device), tanh_norm(width, 20, device, 1.1)
    d = lambda t: t.to(device)
    r, (h,) = ops.gated_residual(d(x), [Branch(Proj(d(a), 0, width), norm=d(wa), scale=0.5, shift=d(shift)),
                                        Branch(Proj(d(b), 0, width), norm=d(wb), scale=0.5)], post=post, norms=[norm], eps=eps,
                                 dtype=dtype)
    mean = (O.rms(av + shift.double(), eps) * wa.double() + O.rms(bv, eps) * wb.double()) / 2
    want = x.double() + f(mean)
    close(r, want, 1e-4, "residual")
    close(h, g(want), TOL[dtype], "norm")
    # one of the two plain
    r, _ = ops.gated_residual(d(x), [Branch(Proj(d(a), 0, width), shift=d(shift), scale=2.0),
                                     Branch(Proj(d(b), 0, width), norm=d(wb))], eps=eps, dtype=dtype, norms=[norm])
    close(r, x.double() + 2 * (av + shift.double()) + O.rms(bv, eps) * wb.double(), 1e-4, "plain and normed")


@on_devices
@in_dtypes
@pytest.mark.parametrize("past", [1, 2, 4, 5, 9])
@pytest.mark.parametrize("width", [64, 35])
def test_depth_average(device, dtype, past, width):
    T = 3
    x, y, rows, coef = rnd(T, width, seed=1), rnd(T, width, seed=2), rnd(past + 2, T, width, seed=3), rnd(past + 1, seed=4)
    norm, g = tanh_norm(width, 10, device)
    rows_d = rows.to(device)
    r, (h,) = ops.gated_residual(x.to(device), [Branch(Proj(y.to(device), 0, width))], norms=[norm], dtype=dtype,
                                 history=History(rows_d, past, coef.to(device)))
    result = x.double() + y.double()
    want = O.depth_average(coef.double(), [*rows[:past].double(), result])
    close(r, want, 1e-5, "average")
    close(h, g(want), TOL[dtype], "norm")
    close(rows_d[past], result, 1e-6, "stored result")
    assert torch.equal(rows_d[past + 1].cpu(), rows[past + 1]) and torch.equal(rows_d[:past].cpu(), rows[:past])
    w = 1 + rnd(width, seed=7)
    _, (h,) = ops.gated_residual(x.to(device), [Branch(Proj(y.to(device), 0, width))], norms=[w.to(device)], eps=1e-4, dtype=dtype,
                                 history=History(rows_d, past, coef.to(device), store=False))
    close(h, O.rms(want, 1e-4) * w.double(), TOL[dtype], "average, then an RMS norm")


@on_devices
def test_embedding_rows_through_a_tanh_norm(device):
    table, ids = rnd(11, 24, seed=1), [3, 0, 10, 3]
    norm, g = tanh_norm(24, 10, device)
    out = torch.zeros((4, 24), device=device)
    r, (h,) = ops.gated_residual(None, ids=i32(ids, device), table=table.bfloat16().to(device), norms=[norm], out=out)
    want = table.bfloat16().double()[ids]
    assert r.data_ptr() == out.data_ptr()
    close(r, want, 1e-6)
    close(h, g(want), TOL[torch.bfloat16])


def test_forms_that_do_not_go_together():
    x, w = rnd(2, 8), torch.ones(8)
    assert [n.kind for n in (Norm(w), Norm(w, w, True), Norm(), Norm(w, w, alpha=1.0))] == [0, 1, 2, 3]
    with pytest.raises(ValueError):
        ops.gated_residual(x, norms=[Norm(w, w, alpha=1.0), w])
    with pytest.raises(ValueError):
        _post_residual(x, [Branch(Proj(x, 0, 8))] * 3, None, None, 1.0, None, None, [], 1, 1e-6, torch.float32, None, None, x, [])
    with pytest.raises(ValueError):
        _post_residual(x, [Branch(Proj(x, 0, 8), Proj(x, 0, 8), w)], None, None, 1.0, None, None, [], 1, 1e-6, torch.float32, None,
                       None, x, [])


# --------------------------------------------------------------------------- feed-forward
@on_devices
@in_dtypes
@pytest.mark.parametrize("form", ["f32", "bf16", "partials"])
def test_xielu(device, dtype, form):
    x = torch.cat([torch.linspace(-12, 12, 480), torch.tensor([0.0, 1e-4, -1e-4, 3e-2, -3e-2, -60.0, 60.0, 1e-8])]).reshape(4, 122)
    x, xv = projection(x, form)
    for p, q in ((0.8, -0.3), (-4.0, 3.0)):
        sp = lambda z: torch.nn.functional.softplus(torch.tensor(z, dtype=torch.float64)).item()
        a = ops.activation(Proj(x.to(device), 2, 120), Act("xielu", sp(p), 0.5 + sp(q)), dtype=dtype)
        want = O.xielu(xv[:, 2:], torch.tensor(p).double(), torch.tensor(q).double())
        err = ((a.double().cpu() - want).abs() / (want.abs() + 1e-3)).max()
        assert err < (2e-4 if dtype == torch.float32 else 8e-3)


@on_devices
@pytest.mark.parametrize("M,N,K", [(200, 136, 72), (640, 520, 264), (130, 100, 40)])
def test_xielu_in_the_epilogue(device, M, N, K):
    x, w = rnd(M, K, seed=1).bfloat16(), rnd(N, K, seed=2, std=2 * K ** -0.5).bfloat16()
    act = torch.tensor([0.4, -0.7], dtype=torch.float64)
    sp = torch.nn.functional.softplus(act).tolist()
    got = ops.linear(x.to(device), w.to(device), swap=False, out_act=Act("xielu", sp[0], 0.5 + sp[1]))
    close(got, O.xielu(x.double() @ w.double().T, act[0], act[1]), 1e-2)


# --------------------------------------------------------------------------- attention
class Pages:
    """Sequences on scattered pages of a small pool."""

    def __init__(self, spec, lens, device, dtype, seed=3):
        self.spec, self.lens, self.device = spec, lens, device
        per = [(n + 31) // 32 for n in lens]
        perm = torch.randperm(sum(per) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
        self.table = torch.zeros((len(lens), max(per)), dtype=torch.int32)
        for b, n in enumerate(per):
            for j in range(n):
                self.table[b, j] = perm.pop()
        pool = lambda d: (50 * rnd(sum(per) + 3, spec.kv_heads, 32, d, seed=9)).to(dtype).to(device)   # what earlier owners left
        self.k, self.v = pool(spec.dim_p), pool(spec.vdim_p)
        self.k[..., spec.dim:] = 0
        self.v[..., spec.vdim:] = 0
        self.table_d = self.table.to(device)

    def slots(self, b, lo, hi):
        return [int(self.table[b, p // 32]) * 32 + p % 32 for p in range(lo, hi)]


def attend(spec, seqs, device, dtype, cuts, sinks=None):
    """seqs: per sequence fp32 (q [T, H, d], k [T, G, d], v [T, G, n]).  cuts: steps, each a list of new-token counts per sequence
    (0: not in the step)."""
    pages = Pages(spec, [len(s[0]) for s in seqs], device, dtype)
    at, out = [0] * len(seqs), [[] for _ in seqs]
    for step in cuts:
        parts = [(b, at[b], at[b] + n) for b, n in enumerate(step) if n]
        cat = lambda i: torch.cat([seqs[b][i][lo:hi].flatten(1) for b, lo, hi in parts])
        q, k, v = (projection(cat(i), form_of(dtype, sum(step)))[0].to(device) for i in range(3))
        pos = i32([p for b, lo, hi in parts for p in range(lo, hi)], device)
        slots = i32([s for b, lo, hi in parts for s in pages.slots(b, lo, hi)], device)
        P = lambda t: Proj(t, 0, t.shape[-1])
        qs = ops.rope_norm_append(spec, P(q), P(k), P(v), None, None, pos, slots, pages.k, pages.v, norm=False)
        ctx = i32([hi for _, _, hi in parts], device)
        rows = pages.table_d[[b for b, _, _ in parts]].contiguous()
        kw = {}
        if any(hi - lo > 1 for _, lo, hi in parts):
            lens = [hi - lo for _, lo, hi in parts]
            kw = dict(q_start=i32([sum(lens[:i]) for i in range(len(lens))], device), q_lens=i32(lens, device), max_q_len=max(lens))
        o = ops.heads_attention(spec, qs, pages.k, pages.v, rows, ctx, sinks=sinks, **kw).float().cpu()
        i = 0
        for b, lo, hi in parts:
            out[b].append(o[i:i + hi - lo])
            i += hi - lo
            at[b] = hi
    return [torch.cat(x) for x in out]


def heads(T, n, d, seed, std=1.0):
    return rnd(T, n, d, seed=seed, std=std).bfloat16().float()


SIZES = [(4, 2, 24, 40), (6, 3, 64, 48), (8, 1, 128, 96), (2, 2, 80, 128), (3, 1, 136, 20), (34, 2, 16, 8)]


@on_devices
@in_dtypes
@pytest.mark.parametrize("H,G,d,n", SIZES)
@pytest.mark.parametrize("cap,window,first", [(4.0, 0, 0), (20.0, 45, 9), (0.0, 33, 40), (2.0, 1, 1), (6.0, 150, 0)])
def test_capped_window_with_kept_first_tokens_and_distances(device, dtype, H, G, d, n, cap, window, first):
    lens = [190, 37, 3]
    r1, r2 = 0.1 + rnd(H, seed=1).abs(), 0.02 + 0.3 * rnd(H, seed=2).abs()
    spec = MapsSpec(H, G, d, n, 2.0 * d ** -0.5, softcap=cap, window=window, keep_first=first, dist_a=r1.to(device),
                    dist_b=r2.to(device), tiled=dtype == torch.bfloat16)
    seqs = [(heads(T, H, d, 10 + i), heads(T, G, d, 20 + i), heads(T, G, n, 30 + i)) for i, T in enumerate(lens)]
    want = []
    for q, k, v in seqs:
        T = len(q)
        mask = O.window_mask(T, window, first) if window else O.causal_mask(T)
        want.append(O.softmax_attention(*(x.double() for x in (q, k, v)), spec.scale, mask, cap,
                                        O.distance_bias(T, r1.double(), r2.double())))
    plans = [[lens], [[130, 2, 1], [1, 30, 2], [59, 5, 0]], [[150, 20, 3]] + [[1, 1, 0]] * 17 + [[1, 0, 0]] * 23]
    for plan in plans:
        for g, w in zip(attend(spec, seqs, device, dtype, plan), want):
            close(g, w, 2e-5 if dtype == torch.float32 else 2.5e-2, f"{plan[0]}")


@on_devices
@in_dtypes
@pytest.mark.parametrize("d", [32, 128])
@pytest.mark.parametrize("edge", [1, 5, 31, 32, 33, 64, 127, 128, 129, 200])
def test_edges_of_a_window_and_of_the_kept_tokens(device, dtype, d, edge):
    """One key stands out; values mark positions.  At distance window - 1 or among the kept tokens it is all a query sees, one
    token further it is not seen."""
    T, first = 330, 7
    window = edge
    spec = MapsSpec(2, 1, d, 16, 1.0, window=window, keep_first=first, softcap=60.0, tiled=dtype == torch.bfloat16)
    q = torch.zeros(T, 2, d)
    q[..., 0] = 6.0
    v = torch.zeros(T, 1, 16)
    v[:, 0, 0] = 1.0
    for place in (first - 1, first, 100):
        k = torch.zeros(T, 1, d)
        k[place, 0, 0] = 6.0                        # a capped score of some 32 against zeros
        vp = v.clone()
        vp[place, 0, 1] = 1.0
        for plan in ([[T]], [[260]] + [[1]] * 12 + [[58]]):
            (o,) = attend(spec, [(q, k, vp)], device, dtype, plan)
            at = torch.arange(T)
            sees = (at >= place) & ((at - place < window) | (place < first))
            close(o[:, 0, 1], sees.double(), 1e-2, f"key {place}, window {window}")
            close(o[:, 1, 0], torch.ones(T, dtype=torch.float64), 1e-2)


@on_devices
@in_dtypes
@pytest.mark.parametrize("H,G,d,n", SIZES)
def test_capped_causal_attention_with_sinks(device, dtype, H, G, d, n):
    lens, cap = [140, 290, 1], 5.0
    sink = rnd(H, seed=4, std=2.0) + 1
    spec = MapsSpec(H, G, d, n, 1.7 * d ** -0.5, softcap=cap, tiled=dtype == torch.bfloat16)
    seqs = [(heads(T, H, d, 10 + i, 1.5), heads(T, G, d, 20 + i), heads(T, G, n, 30 + i)) for i, T in enumerate(lens)]
    want = [O.softmax_attention(*(x.double() for x in s), spec.scale, O.causal_mask(len(s[0])), cap, sink=sink.double()) for s in seqs]
    for plan in ([lens], [[129, 2, 1], [2, 127, 0], [0, 1, 0], [1, 1, 0], [8, 159, 0]]):
        for g, w in zip(attend(spec, seqs, device, dtype, plan, sinks=sink.to(device)), want):
            close(g, w, 2e-5 if dtype == torch.float32 else 2.5e-2)


@on_devices
@in_dtypes
@pytest.mark.parametrize("T", [5, 40])
@pytest.mark.parametrize("H,G,d,n,rot", [(4, 2, 24, 40, 16), (2, 1, 64, 64, 64), (3, 3, 36, 20, 4), (2, 1, 7, 11, 6), (2, 2, 136, 24, 48),
                                         (1, 1, 160, 8, 160), (2, 1, 40, 48, 0)])
@pytest.mark.parametrize("kind", ["bias", "plain", "queries"])
def test_interleaved_rotation_biases_and_append(device, dtype, T, H, G, d, n, rot, kind):
    spec = MapsSpec(H, G, d, n, 1.0, tiled=dtype == torch.bfloat16)
    form, widths = form_of(dtype, T), [H * d, G * d, G * n]
    x = [projection(rnd(T, w, seed=i), form) for i, w in enumerate(widths)]
    bias = rnd(sum(widths), seed=7) if kind == "bias" else None
    table = ops.rope_table(rot, 600, theta=500.0, device=device) if rot else None
    pos, slots = [(37 * i) % 600 for i in range(T)], [(i * 7) % 96 if i != 2 else -1 for i in range(T)]
    kc, vc = (torch.full((3, G, 32, w), 9.0, dtype=dtype, device=device) for w in (spec.dim_p, spec.vdim_p))
    P = [Proj(t.to(device), 0, t.shape[-1]) for t, _ in x]
    q = ops.rope_norm_append(spec, P[0], *((None, None) if kind == "queries" else P[1:]), None if bias is None else bias.to(device),
                             table, i32(pos, device), i32(slots, device), kc, vc, norm=False, interleaved=True)
    full = [v for _, v in x] if bias is None else [v + b.double() for (_, v), b in zip(x, bias.split(widths))]
    # rotate_pairs turns row t by t; pick the rows of the positions asked for
    rotated = lambda a, h: torch.stack([O.rotate_pairs(a[i].view(1, h, d).expand(pos[i] + 1, h, d), 500.0, rot)[-1] for i in range(T)])
    close(q[..., :d], rotated(full[0], H), TOL[dtype], "queries")
    if spec.dim_p > d:
        assert (q[..., d:] == 0).all()
    if kind == "queries":
        assert (kc == 9).all() and (vc == 9).all()
        return
    wk, wv = rotated(full[1], G), full[2].view(T, G, n)
    for i, s in enumerate(slots):
        if s >= 0:
            close(kc[s // 32, :, s % 32, :d], wk[i], 2 * TOL[dtype], "key")
            close(vc[s // 32, :, s % 32, :n], wv[i], 2 * TOL[dtype], "value")
    for s in set(range(96)) - {s for s in slots if s >= 0}:
        assert (kc[s // 32, :, s % 32] == 9).all()


# --------------------------------------------------------------------------- convolution, recurrences
def run_steps(step, lens, cuts):
    """step(parts, decode) -> rows of the parts' tokens; parts: (sequence, first, end).  Returns every sequence's rows."""
    at, out = [0] * len(lens), [[] for _ in lens]
    for cut in cuts:
        parts = [(b, at[b], at[b] + n) for b, n in enumerate(cut) if n]
        decode = all(hi - lo == 1 and lo > 0 for _, lo, hi in parts)
        o, i = step(parts, decode), 0
        for b, lo, hi in parts:
            out[b].append(o[i:i + hi - lo])
            i += hi - lo
            at[b] = hi
    assert at == list(lens)
    return [torch.cat(x) for x in out]


def packed(parts, rows, device):
    lens = [hi - lo for _, lo, hi in parts]
    return (i32([hi for _, _, hi in parts], device), dict(
        q_start=i32([sum(lens[:i]) for i in range(len(lens))], device), q_lens=i32(lens, device),
        rows=i32([rows[b] for b, _, _ in parts], device)))


LENS = [150, 41, 6, 1]
PLANS = {"whole": [LENS], "portions": [[2, 0, 1, 1], [17, 16, 2, 0], [1, 2, 1, 0], [2, 22, 2, 0], [128, 1, 0, 0]],
         "single tokens": [[130, 20, 3, 1]] + [[1, 1, 1, 0]] * 3 + [[1, 1, 0, 0]] * 17 + [[0, 1, 0, 0]]}
ROWS = [4, 0, 5, 2]                  # slots; 1 and 3 belong to nobody


@on_devices
@in_dtypes
@pytest.mark.parametrize("taps,C,bias", [(1, 24, True), (2, 16, False), (3, 40, True), (4, 1032, False), (5, 30, True), (8, 64, True)])
def test_short_convolution(device, dtype, taps, C, bias):
    w, b = rnd(taps, C, seed=1), rnd(C, seed=2) if bias else None
    xs = [rnd(n, C, seed=3 + i).bfloat16().float() for i, n in enumerate(LENS)]
    conv = ShortConv(w.to(device), None if b is None else b.to(device))
    state = torch.full((6, taps, C), 1e3, device=device)       # a slot needs no clearing

    def step(parts, decode):
        ctx, kw = packed(parts, ROWS, device)
        x = projection(torch.cat([xs[s][lo:hi] for s, lo, hi in parts]), form_of(dtype, len(parts) if decode else 99))[0]
        return ops.short_conv(Proj(x.to(device), 0, C), conv, state, ctx, dtype=dtype, **kw).float().cpu()

    for name in ("whole", "portions"):
        for x, g in zip(xs, run_steps(step, LENS, PLANS[name])):
            close(g, O.silu(O.short_conv(x.double(), w.double().T, None if b is None else b.double())), TOL[dtype], name)
    assert (state[[1, 3]] == 1e3).all()


@on_devices
@in_dtypes
@pytest.mark.parametrize("H,G,d,n,taps,decay,strength", [
    (4, 2, 16, 24, 3, 0.0, 0.0), (2, 2, 64, 64, 4, -3.0, 3.0), (3, 1, 128, 72, 2, -6.0, 0.0), (6, 3, 24, 128, 1, 2.0, 0.0),
    (2, 1, 7, 11, 5, -2.0, -3.0), (1, 1, 200, 40, 4, -4.0, 1.0), (4, 4, 32, 8, 3, -8.0, 6.0), (2, 2, 72, 16, 8, 5.0, 0.0)])
@pytest.mark.parametrize("plan", PLANS)
def test_gated_delta_rule(device, dtype, H, G, d, n, taps, decay, strength, plan):
    """Decays from almost none to almost all of the state, weak and full writes."""
    C, D = 2 * G * d + H * n, lambda t: t.to(device)
    rate, dtb = torch.exp(rnd(H, seed=1) + decay), rnd(H, seed=2)
    w, norm = rnd(taps, C, seed=3, std=taps ** -0.5), 1 + 0.3 * rnd(n, seed=4)
    draw = lambda width, seed, shift=0.0: [rnd(T, width, seed=seed + i).bfloat16().float() + shift for i, T in enumerate(LENS)]
    xs, decays, strengths, gates = draw(C, 10), draw(H, 30), draw(H, 40, strength), draw(H * n, 50)
    rec = HeadRecurrence(H, G, d, n, 0, G * d, 2 * G * d, D(rate), D(dtb), delta=True, q_scale=d ** -0.5, eps=1e-4)
    conv = ShortConv(D(w))
    state, ring = torch.full((6, *rec.state_shape), 1e3, device=device), torch.full((6, taps, C), 1e3, device=device)

    def step(parts, decode):
        ctx, kw = packed(parts, ROWS, device)
        form = form_of(dtype, 1 if decode else 99)
        pick = lambda ts: projection(torch.cat([ts[s][lo:hi] for s, lo, hi in parts]), form)[0].to(device)
        x, a, b, g = (Proj(t, 0, t.shape[-1]) for t in map(pick, (xs, decays, strengths, gates)))
        if decode:
            kw = dict(rows=kw["rows"])
        return ops.head_recurrence(rec, x, conv, a, b, g, D(norm), state, ring, ctx, dtype=dtype, **kw).float().cpu()

    got = run_steps(step, LENS, PLANS[plan])
    pick = torch.arange(H) // (H // G)
    for i, T in enumerate(LENS):
        y = O.silu(O.short_conv(xs[i].double(), w.double().T))
        q, k, v = y.split([G * d, G * d, H * n], -1)
        q, k = (O.unit(t.reshape(T, G, d))[:, pick] for t in (q, k))
        g = torch.exp(-rate.double() * O.softplus(decays[i].double() + dtb.double()))
        o = O.delta_rule(q * d ** -0.5, k, v.reshape(T, H, n), g, torch.sigmoid(strengths[i].double()))
        near(got[i], (O.rms(o, 1e-4) * norm.double()).reshape(T, -1) * O.silu(gates[i].double()), dtype, f"sequence {i}")
    assert (state[[1, 3]] == 1e3).all() and (ring[[1, 3]] == 1e3).all()


@on_devices
@in_dtypes
@pytest.mark.parametrize("H,G,N,n,taps,parts,decay", [
    (4, 2, 16, 24, 4, 2, 0.0), (2, 1, 128, 64, 4, 1, -3.0), (6, 6, 64, 40, 2, 3, -6.0), (3, 1, 7, 11, 3, 1, -2.0),
    (4, 1, 24, 8, 1, 16, 3.0), (2, 2, 160, 136, 5, 4, -5.0), (8, 2, 32, 128, 4, 2, -4.0), (12, 3, 8, 5, 3, 12, 0.0)])
@pytest.mark.parametrize("plan", PLANS)
def test_state_space_mixer(device, dtype, H, G, N, n, taps, parts, decay, plan):
    inner, D = H * n, lambda t: t.to(device)
    C = inner + 2 * G * N
    A, dtb, skip = torch.exp(rnd(H, seed=1) + decay), rnd(H, seed=2), rnd(H, seed=5)
    w, cb, norm = rnd(taps, C, seed=3, std=taps ** -0.5), rnd(C, seed=6), 1 + 0.3 * rnd(inner, seed=4)
    draw = lambda width, seed: [rnd(T, width, seed=seed + i).bfloat16().float() for i, T in enumerate(LENS)]
    xs, dts, zs = draw(C, 10), draw(H, 30), draw(inner, 50)
    rec = HeadRecurrence(H, G, N, n, inner + G * N, inner, 0, D(A), D(dtb), delta=False, skip=D(skip), eps=1e-4)
    conv = ShortConv(D(w), D(cb))
    state, ring = torch.full((6, *rec.state_shape), 1e3, device=device), torch.full((6, taps, C), 1e3, device=device)

    def step(parts_, decode):
        ctx, kw = packed(parts_, ROWS, device)
        form = form_of(dtype, 1 if decode else 99)
        x, a, g = (projection(torch.cat([ts[s][lo:hi] for s, lo, hi in parts_]), form)[0].to(device) for ts in (xs, dts, zs))
        if decode:
            kw = dict(rows=kw["rows"])
        P = lambda t: Proj(t, 0, t.shape[-1])
        return ops.head_recurrence(rec, P(x), conv, P(a), None, P(g), D(norm), state, ring, ctx, parts=parts, dtype=dtype,
                                   **kw).float().cpu()

    got = run_steps(step, LENS, PLANS[plan])
    pick = torch.arange(H) // (H // G)
    for i, T in enumerate(LENS):
        y = O.silu(O.short_conv(xs[i].double(), w.double().T, cb.double()))
        x, B, Cc = y.split([inner, G * N, G * N], -1)
        x = x.reshape(T, H, n)
        dt = O.softplus(dts[i].double() + dtb.double())
        o = O.state_space(x, B.reshape(T, G, N)[:, pick], Cc.reshape(T, G, N)[:, pick], dt, -A.double())
        o = (o + skip.double()[:, None] * x).reshape(T, -1) * O.silu(zs[i].double())
        near(got[i], O.rms(o.view(T, parts, -1), 1e-4).reshape(T, -1) * norm.double(), dtype, f"sequence {i}")
    assert (state[[1, 3]] == 1e3).all() and (ring[[1, 3]] == 1e3).all()


@on_devices
@in_dtypes
def test_a_write_survives_hundreds_of_tokens(device, dtype):
    """Delta rule without decay: a key written once is read back after 600 other writes to an orthogonal key."""
    T, d, n = 601, 16, 16
    x = torch.zeros(T, 2 * d + n)
    x[0, d], x[1:, d + 1] = 20.0, 20.0                                 # key 0, then key 1
    x[-1, 0] = 20.0                                                    # the last query asks for key 0
    x[:, :d] += 1e-3
    x[0, 2 * d], x[1:, 2 * d + 1] = 3.0, 3.0
    D = lambda t: t.to(device)
    rec = HeadRecurrence(1, 1, d, n, 0, d, 2 * d, D(torch.full((1,), 1e-7)), D(torch.zeros(1)), delta=True, eps=1e-6)
    state, ring = torch.zeros((1, *rec.state_shape), device=device), torch.zeros((1, 1, 2 * d + n), device=device)
    conv, norm = ShortConv(D(torch.ones(1, 2 * d + n))), D(torch.ones(n))
    outs = []
    for lo, hi in ((0, 300), (300, 590), *((t, t + 1) for t in range(590, T))):
        kw = {} if hi - lo == 1 else dict(q_start=i32([0], device), q_lens=i32([hi - lo], device))
        c = lambda v: Proj(v.to(device=device, dtype=dtype if hi - lo > 1 else torch.float32), 0, v.shape[1])
        outs.append(ops.head_recurrence(rec, c(x[lo:hi]), conv, c(torch.zeros(hi - lo, 1)), c(torch.full((hi - lo, 1), 8.0)),
                                        c(torch.ones(hi - lo, n)), norm, state, ring, i32([hi], device), dtype=dtype, **kw))
    o = torch.cat(outs).float().cpu()
    assert o[-1, 0] > 20 * o[-1, 1].abs()
    assert (o[-2, 0] - o[-2, 1]).abs() < 0.1                           # a query between the two keys reads both


@on_devices
@in_dtypes
def test_inactive_rows_of_a_step_are_left_alone(device, dtype):
    H, d, n = 2, 8, 8
    rec = HeadRecurrence(H, H, d, n, 0, H * d, 2 * H * d, torch.ones(H, device=device), torch.zeros(H, device=device), delta=True)
    C = 2 * H * d + H * n
    state, ring = rnd(3, *rec.state_shape).to(device), rnd(3, 4, C).to(device)
    before = state.clone(), ring.clone()
    conv = ShortConv(rnd(4, C, seed=1).to(device))
    P = lambda w, s: Proj(rnd(3, w, seed=s).to(device), 0, w)
    out = ops.head_recurrence(rec, P(C, 2), conv, P(H, 3), P(H, 4), P(H * n, 5), torch.ones(n, device=device), state, ring,
                              i32([7, -1, 5], device), dtype=dtype)
    assert (out[0] != 0).any()
    assert torch.equal(state[1], before[0][1]) and torch.equal(ring[1], before[1][1])
    assert not torch.equal(state[0], before[0][0])
    assert (ring[0] != before[1][0]).any(-1).tolist() == [False, False, True, False]     # position 6 in a ring of four


@on_devices
@in_dtypes
@pytest.mark.parametrize("W,parts", [(96, 1), (96, 3), (70, 5), (2048, 8), (2048, 16), (2048, 1), (40, 40), (12288, 1), (1056, 1)])
def test_gated_group_norm(device, dtype, W, parts):
    y, w = rnd(5, W, seed=1).to(dtype), 1 + rnd(W, seed=2)
    y[1] *= 1e-2
    for form in ("f32", "bf16", "partials"):
        g, gv = projection(rnd(5, W + 8, seed=3), form)
        got = ops.gated_group_norm(y.to(device), Proj(g.to(device), 8, W), "silu", w.to(device), parts, 1e-3, dtype)
        z = (y.double() * O.silu(gv[:, 8:])).view(5, parts, -1)
        close(got, O.rms(z, 1e-3).reshape(5, W) * w.double(), TOL[dtype])
