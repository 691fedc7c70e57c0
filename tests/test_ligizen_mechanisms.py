"""Each mechanism of the parallel layer-by-layer decoders against the plain statement in ligizen_oracle.py: the operators'
PyTorch form on the CPU and the kernels on a GPU, in 32-bit and in bfloat16."""
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import ligizen_oracle as O  # noqa: E402

from nkipy_b200 import ops  # noqa: E402
from nkipy_b200.models.config import ClampedSpec, ExpertsSpec, RopeSpec, rope_frequencies  # noqa: E402
from nkipy_b200.models.mixers import Tensors  # noqa: E402
from nkipy_b200.models.moe import RoutedExperts  # noqa: E402
from nkipy_b200.ops import Branch, LatentSpec, MapsSpec, Norm, Proj  # noqa: E402

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
@on_devices
@in_dtypes
@pytest.mark.parametrize("form", ["f32", "bf16", "partials"])
@pytest.mark.parametrize("width", [96, 70, 2052])
def test_layer_norm_and_copy_of_a_residual(device, dtype, form, width):
    T, eps = 5, 1e-4
    x, w, b = rnd(T, width, seed=1) + 3, 1 + rnd(width, seed=2), rnd(width, seed=3)
    y, yv = projection(rnd(T, width, seed=4), form)
    d = lambda t: t.to(device)
    want = x.double() + yv
    r, (h,) = ops.gated_residual(d(x), [Branch(Proj(d(y), 0, width))], norms=[Norm(d(w), d(b), True)], eps=eps, dtype=dtype)
    close(r, want, 1e-5, "residual")
    close(h, O.layer_norm(want, w.double(), b.double(), eps), TOL[dtype], "layer norm")
    r, (h,) = ops.gated_residual(d(x), [Branch(Proj(d(y), 0, width))], norms=[Norm()], dtype=dtype)
    close(h, want, TOL[dtype], "copy")
    with pytest.raises(ValueError):
        ops.gated_residual(d(x), norms=[Norm(), d(w)])


@on_devices
@in_dtypes
@pytest.mark.parametrize("form", ["f32", "bf16", "partials"])
@pytest.mark.parametrize("width", [96, 70, 2048])
def test_normed_branch(device, dtype, form, width):
    """The smallest rows matter: the epsilon is inside the root."""
    T, eps = 6, 1e-3
    x, w = rnd(T, width, seed=1), 1 + rnd(width, seed=2)
    scale = torch.tensor([1e-3, 1e-2, 0.1, 1.0, 10.0, 0.0])[:, None]
    y, yv = projection(rnd(T, width, seed=4) * scale, "f32" if form == "partials" else form)
    if form == "partials":
        y = torch.stack([0.25 * y, 0.75 * y])
    norm = [Norm(torch.ones(width, device=device), torch.zeros(width, device=device), True)]
    r, _ = ops.gated_residual(x.to(device), [Branch(Proj(y.to(device), 0, width), norm=w.to(device))], norms=norm, eps=eps, dtype=dtype)
    close(r, x.double() + O.rms(yv, eps) * w.double(), 2e-5)


@on_devices
@in_dtypes
@pytest.mark.parametrize("form", ["f32", "bf16", "partials"])
@pytest.mark.parametrize("width", [96, 70])
def test_three_branches_with_unweighted_rows_and_one_gate_per_token(device, dtype, form, width):
    T, k = 7, 3
    x, w, b = rnd(T, width, seed=1), 1 + rnd(width, seed=2), rnd(width, seed=3)
    m, mv = projection(rnd(T, width + 4, seed=4), form)
    s, sv = projection(rnd(T, width, seed=5), form)
    g, gv = projection(rnd(T, 9, seed=6, std=2.0), "f32" if form == "bf16" else form)
    rows = rnd(T * k, width, seed=7)
    pos = torch.randperm(T * k, generator=torch.Generator().manual_seed(5)).to(torch.int32)
    pos[4] = -1
    routed = torch.zeros(T, width, dtype=torch.float64)
    for i, q in enumerate(pos.tolist()):
        if q >= 0:
            routed[i // k] += rows[q].double()
    d = lambda t: t.to(device)
    want = x.double() + mv[:, 4:] + routed + torch.sigmoid(gv[:, 8:]) * sv
    r, (h,) = ops.gated_residual(
        d(x), [Branch(Proj(d(m), 4, width)), Branch(Proj(d(rows), 0, width), pair_pos=d(pos), top_k=k),
               Branch(Proj(d(s), 0, width), Proj(d(g), 8, 1))], norms=[Norm(d(w), d(b), True)], eps=1e-5, dtype=dtype)
    close(r, want, 1e-5, "residual")
    close(h, O.layer_norm(want, w.double(), b.double(), 1e-5), TOL[dtype], "norm")


# --------------------------------------------------------------------------- activations
@on_devices
@in_dtypes
@pytest.mark.parametrize("form", ["f32", "bf16", "partials"])
@pytest.mark.parametrize("n", [24, 31])
def test_clamped_gate_on_both_sides_of_its_limit(device, dtype, form, n):
    y, v = projection(rnd(6, 2 * n + 8, std=2.5), form)
    g, u = v[:, 8:8 + n], v[:, 8 + n:]
    for limit in (0.7, 1.9, 100.0):
        eye = torch.eye(n, dtype=torch.float64)
        h = torch.cat([g, u], 1)
        zero = torch.zeros(n, n, dtype=torch.float64)
        want = O.clamped_mlp(h, torch.cat([eye, zero], 1), torch.cat([zero, eye], 1), eye, limit)
        got = ops.gated_act(Proj(y.to(device), 8, n), Proj(y.to(device), 8 + n, n), "clamped", dtype=dtype, limit=limit)
        close(got, want, TOL[dtype], f"limit {limit}")


@on_devices
@in_dtypes
@pytest.mark.parametrize("n,layer", [(24, 1), (9, 2)])
def test_activation_times_rows_of_a_table(device, dtype, n, layer):
    T, vocab = 11, 13
    z, zv = projection(rnd(T, n, std=2.0), "partials")
    table = rnd(vocab, 3 * n, seed=1).to(dtype)
    ids = i32([0, 12, 5, 5, 3, 1, 7, 0, 2, 11, 12], device)
    got = ops.gated_act(Proj(z.to(device), 0, n), Proj(table.to(device), layer * n, n), "gelu_tanh", dtype=dtype, up_rows=ids)
    close(got, O.gelu_tanh(zv) * table.double()[ids.cpu().long(), layer * n:(layer + 1) * n], TOL[dtype])


@on_devices
@pytest.mark.parametrize("rows,vocab", [(3, 64), (2, 61)])
def test_logits_are_capped(device, rows, vocab):
    z = rnd(rows, vocab, std=40.0)
    want = O.softcap(z.double(), 25.0)
    close(ops.softcap(z.to(device), 25.0), want, 1e-6)


@on_devices
@in_dtypes
@pytest.mark.parametrize("H,n", [(3, 40), (2, 33), (5, 264), (1, 8)])
def test_one_gate_per_head(device, dtype, H, n):
    T = 9
    x = rnd(H, T, n).to(dtype)
    for form in ("bf16" if dtype == torch.bfloat16 else "f32", "partials"):
        g, gv = projection(rnd(T, H + 3, seed=1, std=2.0), form)
        got = ops.gate_heads(x.to(device).transpose(0, 1), Proj(g.to(device), 3, H), "sigmoid")
        close(got, (x.double().transpose(0, 1) * torch.sigmoid(gv[:, 3:])[..., None]).reshape(T, -1), TOL[dtype], form)


# --------------------------------------------------------------------------- experts
@on_devices
@pytest.mark.parametrize("form", ["f32", "partials"])
@pytest.mark.parametrize("E,top", [(6, 2), (40, 1), (70, 9), (3, 3)])
def test_sigmoid_router_keeps_the_scores(device, form, E, top):
    T = 33
    z, zv = projection(rnd(T, E + 7, std=2.0), form)
    w, e = ops.router_topk(Proj(z.to(device), 5, E), top, "sigmoid_topk")
    for t in range(T):
        pick, score = O.route(zv[t, 5:5 + E], top)
        assert e[t].tolist() == pick
        close(w[t], score, 1e-6)


@on_devices
@in_dtypes
@pytest.mark.parametrize("T,width", [(5, 40), (70, 33), (3000, 24)])
def test_dispatch_scales_the_rows_it_gathers(device, dtype, T, width):
    E, k = 7, 3
    x = rnd(T, width).to(dtype)
    experts = torch.stack([torch.randperm(E, generator=torch.Generator().manual_seed(t))[:k] for t in range(T)]).to(torch.int32)
    w = torch.rand(T, k, generator=torch.Generator().manual_seed(1))
    plan = ops.moe_dispatch(x.to(device), experts.to(device), 0, E, weights=w.to(device))
    pos = plan.pair_pos.cpu().long().reshape(T, k)
    assert sorted(pos.reshape(-1).tolist()) == list(range(T * k))
    close(plan.x_sorted.cpu()[pos], w.double()[..., None] * x.double()[:, None], 1e-6 if dtype == torch.float32 else 5e-3)


@on_devices
@in_dtypes
@pytest.mark.parametrize("W,ff,E,top,tokens,shared", [(64, 40, 6, 2, 50, 48), (64, 40, 6, 1, 3, None), (70, 33, 5, 3, 20, 9),
                                                      (128, 64, 40, 4, 300, 64)])
def test_routed_experts_scale_their_input(device, dtype, W, ff, E, top, tokens, shared):
    """Clamps that bite make the weight on the input differ from the weight on the output."""
    ws = {"router": rnd(E, W, seed=1, std=4 / W ** 0.5)}
    for e in range(E):
        for i, n in enumerate(("gate", "up", "down")):
            ws[f"e{e}.{n}"] = rnd(*((W, ff) if n == "down" else (ff, W)), seed=10 * e + i + 2, std=2 * W ** -0.5)
    m = {"router": {"experts": E, "top": top}, "expert": {"ff": ff, "limit": 0.9}}
    if shared:
        m["shared"] = {"ff": shared, "limit": 0.6}
        ws["shared.sg"] = rnd(1, W, seed=900, std=2 * W ** -0.5)
        for i, n in enumerate(("gate", "up", "down")):
            ws["shared." + n] = rnd(*((W, shared) if n == "down" else (shared, W)), seed=901 + i, std=2 * W ** -0.5)
    ws = {k: v.bfloat16() for k, v in ws.items()}
    spec = ExpertsSpec(E, top, ff, score="sigmoid", limit=0.9, scale_input=True, shared=ClampedSpec(shared, 0.6) if shared else None)
    block = RoutedExperts(spec, Tensors(lambda k: ws[k].to(device), "", dtype))
    h = rnd(tokens, W, seed=99).to(dtype)

    class Model:
        project = staticmethod(lambda x, w: ops.linear(x, w) if x.dtype == torch.float32 else ops.linear(x, w, fp32_out=True))

    got = ops.gated_residual(torch.zeros(tokens, W, device=device), block.run(Model, h.to(device)))[0].cpu()
    want = O.experts(h.double(), {k: v.double() for k, v in ws.items()}, m)
    bad = ((got.double() - want).abs().amax(-1) / want.abs().max()) > (1e-4 if dtype == torch.float32 else 3e-2)
    assert bad.sum() <= (0 if dtype == torch.float32 else tokens // 50)          # a tie in the router may fall the other way


# --------------------------------------------------------------------------- rotation
@pytest.mark.parametrize("dims,base,scaling", [(64, 50000.0, (8.0, 1.0, 4.0, 1024)), (48, 300.0, (4.0, 2.0, 3.0, 40)),
                                               (6, 10000.0, (2.0, 1.0, 32.0, 8192))])
def test_frequency_bands(dims, base, scaling):
    factor, low, high, original = scaling
    freq, mult = rope_frequencies(RopeSpec(base, dims, factor, original, low=low, high=high))
    plain, _ = rope_frequencies(RopeSpec(base, dims))
    want = O.band_scaled(plain, dict(factor=factor, low=low, high=high, original=original))
    assert mult == 1.0 and torch.allclose(freq, want, rtol=1e-12)
    assert (freq / plain).min() < 0.999 and freq[0] == plain[0]


def rope(rot, positions, device):
    f, mult = rope_frequencies(RopeSpec(rot["base"], rot["dims"]))
    return ops.rope_table(rot["dims"], positions, inv_freq=f, scaling=mult, device=device)


@on_devices
@in_dtypes
@pytest.mark.parametrize("own", [True, False])
@pytest.mark.parametrize("H,G,d,n,dims", [(4, 2, 24, 40, 16), (3, 1, 64, 64, 64), (2, 2, 136, 144, 96), (2, 1, 7, 11, 6),
                                          (5, 5, 128, 72, 32), (1, 1, 300, 20, 300)])
def test_biases_rotation_norm_and_append(device, dtype, own, H, G, d, n, dims):
    T, eps, rot = 11, 1e-2, {"base": 50.0, "dims": dims}
    widths = [H * d, G * d, G * n] if own else [H * d]
    y, v = projection(rnd(T, sum(widths) + 8, std=0.3), form_of(dtype, T))
    bias = rnd(sum(widths), seed=3, std=0.3)
    s = MapsSpec(H, G, d, n, 1.0, maps=1, eps=eps, tiled=dtype == torch.bfloat16)
    kc = torch.full((3, G, 32, s.dim_p), 7.0, dtype=dtype, device=device)
    vc = torch.full((3, G, 32, s.vdim_p), 7.0, dtype=dtype, device=device)
    pos = [40, 0, 1, 2, 90, 33, 34, 5, 63, 64, 17]
    slots = [65, 3, 4, 5, -1, 0, 31, 32, 95, 64, 50]
    cols, c = [], 8
    for w in widths:
        cols.append(Proj(y.to(device), c, w))
        c += w
    q = ops.rope_norm_append(s, *(cols if own else cols + [None, None]), bias.to(device), rope(rot, 100, device), i32(pos, device),
                             i32(slots, device), kc, vc)
    x = v[:, 8:] + bias.double()
    a = O.angles(100, rot)[pos]
    head = lambda z, m: O.rms(O.rotate_half(z.reshape(T, m, d), a), eps)
    close(q[..., :d], head(x[:, :H * d], H), TOL[dtype], "queries")
    assert (q[..., d:] == 0).all()
    if not own:
        assert (kc == 7).all() and (vc == 7).all()
        return
    k, val = head(x[:, H * d:(H + G) * d], G), x[:, (H + G) * d:].reshape(T, G, n)
    seen = torch.zeros(96, dtype=torch.bool)
    for t, slot in enumerate(slots):
        if slot >= 0:
            seen[slot] = True
            close(kc[slot // 32, :, slot % 32, :d], k[t], TOL[dtype], "keys")
            close(vc[slot // 32, :, slot % 32, :n], val[t], TOL[dtype], "values")
    assert (kc.cpu().permute(0, 2, 1, 3).reshape(96, -1)[~seen] == 7).all()


# --------------------------------------------------------------------------- chunked attention
class Paged:
    """Blocks of several sequences in a shuffled pool; rows of a sequence's tokens are written and read through its table."""

    def __init__(self, lens, device, seed=0):
        self.lens, self.device = lens, device
        self.pages = [(n + 31) // 32 for n in lens]
        self.total = sum(self.pages) + 2
        perm = torch.randperm(self.total, generator=torch.Generator().manual_seed(seed))
        self.table, at = torch.zeros(len(lens), max(self.pages), dtype=torch.int32), 0
        for b, p in enumerate(self.pages):
            self.table[b, :p] = perm[at:at + p].int()
            at += p

    def pool(self, heads, width, rows, dtype):
        """rows: per sequence [T, heads, n] -> [blocks, heads, 32, width], unused places hold large values."""
        out = torch.full((self.total, heads, 32, width), 30.0)
        for b, x in enumerate(rows):
            for t in range(x.shape[0]):
                out[self.table[b, t // 32], :, t % 32] = torch.nn.functional.pad(x[t], (0, width - x.shape[-1]))
        return out.to(dtype).to(self.device)


def attend_all(c, news, run):
    """run(q_start, q_lens, context_lens, max_q_len) over the last news[b] tokens of every sequence."""
    d = c.device
    start = [sum(news[:i]) for i in range(len(news))]
    return run(i32(start, d), i32(news, d), i32(c.lens, d), max(news))


@on_devices
@in_dtypes
@pytest.mark.parametrize("H,G,d,n", [(4, 2, 24, 40), (6, 1, 64, 64), (3, 3, 128, 96), (2, 1, 136, 144), (34, 2, 8, 8)])
@pytest.mark.parametrize("chunk", [1, 21, 64, 97, 1000])
def test_chunked_attention(device, dtype, H, G, d, n, chunk):
    """One key of each sequence stands out; queries just inside and just outside its chunk."""
    lens = [200, 33, 98]
    c = Paged(lens, device)
    s = MapsSpec(H, G, d, n, d ** -0.5, maps=1, chunk=chunk, tiled=dtype == torch.bfloat16)
    q, k, v = ([rnd(T, m, w, seed=7 * i + j).to(dtype) for i, T in enumerate(lens)]
               for j, (m, w) in enumerate(((H, d), (G, d), (G, n))))
    for i, T in enumerate(lens):
        far = min(T - 1, (T - 1) // chunk * chunk)
        for at in {far, max(0, far - 1)}:                  # the first key of the last chunk, and the one before it
            k[i][at] = (4 * q[i][-1].float().reshape(G, H // G, d).mean(1)).to(dtype)
            v[i][at] = 5.0 if at == far else -5.0
    want = [O.attend(a.double(), b.double(), w.double(), d ** -0.5, O.chunk_mask(T, chunk)) for a, b, w, T in zip(q, k, v, lens)]
    kc, vc = c.pool(G, s.dim_p, k, dtype), c.pool(G, s.vdim_p, v, dtype)
    if dtype == torch.bfloat16:                            # places beyond a sequence's end hold numbers, never NaN
        assert torch.isfinite(kc).all()
    pad = lambda x: torch.nn.functional.pad(x, (0, s.dim_p - d)).to(device).contiguous()
    table = c.table.to(device)
    for news in (lens, [60, 33, 2], [2, 1, 98], [1, 1, 1]):
        qs = pad(torch.cat([x[-m:] for x, m in zip(q, news)]))
        got = attend_all(c, news, lambda a, b, e, m: ops.heads_attention(s, qs, kc, vc, table, e, q_start=a, q_lens=b, max_q_len=m))
        close(got, torch.cat([w[-m:] for w, m in zip(want, news)]), TOL[dtype], f"{news}")
    for splits in (1, 3):
        got = ops.heads_attention(s, pad(torch.stack([x[-1] for x in q])), kc, vc, table, i32(lens, device), num_splits=splits)
        close(got, torch.stack([w[-1] for w in want]), TOL[dtype], "decode")


# --------------------------------------------------------------------------- latent attention
# heads, dim, rot, vdim, rank, q_rank: the four row sizes of the tensor-core kernel, odd sizes, sizes beyond it
LATENT = [(4, 20, 8, 24, 40, 56), (18, 64, 24, 72, 128, 264), (3, 128, 64, 128, 200, 72), (33, 32, 64, 40, 512, 40),
          (3, 5, 6, 7, 13, 11), (2, 136, 72, 136, 72, 48), (2, 24, 16, 16, 600, 2056)]


def latent_case(H, d, r, n, R, Q, dtype, window, eps=1e-3):
    return LatentSpec(H, d, r, n, R, Q, 1.5 * (d + r) ** -0.5, window, eps, tiled=dtype == torch.bfloat16)


@on_devices
@in_dtypes
@pytest.mark.parametrize("sizes", LATENT)
def test_latents_are_normed_rotated_and_cached(device, dtype, sizes):
    H, d, r, n, R, Q = sizes
    s, rot, T = latent_case(*sizes, dtype, 0), {"base": 40.0, "dims": r}, 9
    for form in ("f32", "partials") + (("bf16",) if dtype == torch.bfloat16 else ()):
        y, v = projection(rnd(T, Q + R + r + 8, std=0.1), form)
        qn, kn = 1 + rnd(Q, seed=1), 1 + rnd(R, seed=2)
        cache = torch.full((3, 1, 32, s.row), 7.0, dtype=dtype, device=device)
        pos, slots = [40, 0, 1, 2, 90, 33, 34, 5, 63], [65, 3, 4, 5, -1, 0, 31, 32, 95]
        table = rope(rot, 100, device)
        c = ops.latent_append(s, Proj(y.to(device), 8, Q), Proj(y.to(device), 8 + Q, R + r), qn.to(device), kn.to(device), table,
                              i32(pos, device), i32(slots, device), cache)
        x = v[:, 8:]
        close(c, O.rms(x[:, :Q], s.eps) * qn.double(), TOL[dtype], "query latent")
        a = O.angles(100, rot)[pos]
        row = torch.cat([O.rms(x[:, Q:Q + R], s.eps) * kn.double(), O.rotate_pairs(x[:, None, Q + R:], a)[:, 0]], 1)
        flat = cache.cpu().reshape(96, s.row)
        for t, slot in enumerate(slots):
            if slot >= 0:
                close(flat[slot, :R], row[t, :R], TOL[dtype], "latent")
                close(flat[slot, R:R + r], row[t, R:], TOL[dtype], "rotated part")
                assert (flat[slot, R + r:] == 0).all()
        rest = [i for i in range(96) if i not in slots]
        assert (flat[rest] == 7).all()
        pages = i32([2, 0], device)
        lat, rk = ops.latent_gather(s, cache, pages, (r + 7) // 8 * 8)
        assert torch.equal(lat.cpu(), cache.cpu()[[2, 0], 0].reshape(64, -1)[:, :R])
        assert torch.equal(rk.cpu()[:, :r], cache.cpu()[[2, 0], 0].reshape(64, -1)[:, R:R + r])


@on_devices
@in_dtypes
@pytest.mark.parametrize("sizes", LATENT)
@pytest.mark.parametrize("form", ["finished", "partials"])
def test_queries_are_split_and_rotated(device, dtype, sizes, form):
    H, d, r, n, R, Q = sizes
    s, rot, T = latent_case(*sizes, dtype, 0), {"base": 40.0, "dims": r}, 9
    y, v = projection(rnd(T, H * (d + r)), form if form == "partials" else ("bf16" if dtype == torch.bfloat16 else "f32"))
    pos = [40, 0, 1, 2, 90, 33, 34, 5, 63]
    x = v.reshape(T, H, d + r)
    rotated = O.rotate_pairs(x[..., d:], O.angles(100, rot)[pos])
    plain = torch.full((H, T, d), 7.0, dtype=dtype, device=device)
    q = torch.full((H, T, s.row), 7.0, dtype=dtype, device=device)
    ops.latent_queries(s, Proj(y.to(device), 0, H * (d + r)), rope(rot, 100, device), i32(pos, device), plain.transpose(0, 1),
                       q.transpose(0, 1)[..., R:])
    close(plain.transpose(0, 1), x[..., :d], TOL[dtype])
    close(q.transpose(0, 1)[..., R:R + r], rotated, TOL[dtype])
    assert (q[..., R + r:] == 0).all() and (q[..., :R] == 7).all()


@on_devices
@in_dtypes
@pytest.mark.parametrize("H,T,K,N,pad", [(4, 3, 24, 40, 8), (2, 70, 128, 512, 64), (3, 5, 7, 11, 2), (5, 1, 64, 33, 0)])
def test_products_per_head(device, dtype, H, T, K, N, pad):
    x, w = rnd(H, T, K).to(dtype), rnd(H, N, K, seed=1).to(dtype)
    want = torch.einsum("htk,hnk->htn", x.double(), w.double())
    close(ops.head_linear(x.to(device), w.to(device)), want, TOL[dtype])
    wide = torch.full((H, T, N + pad), 7.0, dtype=dtype, device=device)
    ops.head_linear(x.to(device), w.to(device), out=wide[..., :N])
    close(wide[..., :N], want, TOL[dtype])
    assert (wide[..., N:] == 7).all()


class Latent:
    """Queries and cached rows of several sequences; the key a window before the last token, and the one before that, score high."""

    def __init__(self, sizes, dtype, device, lens, window, sinks=True):
        H, d, r, n, R, Q = sizes
        self.s, self.lens, self.device, self.dtype = latent_case(*sizes, dtype, window), lens, device, dtype
        self.c = Paged(lens, device)
        self.uk, self.uv = rnd(H, d, R, seed=1, std=R ** -0.5).to(dtype), rnd(H, n, R, seed=2, std=R ** -0.5).to(dtype)
        self.sinks = rnd(H, seed=3) + 1 if sinks else None
        self.q = [rnd(T, H, d + r, seed=10 + i).to(dtype) for i, T in enumerate(lens)]
        self.rows = [rnd(T, R + r, seed=30 + i).to(dtype) for i, T in enumerate(lens)]
        for i, T in enumerate(lens):
            last = self.q[i][-1].float().mean(0)
            for at, size in ((T - window, 3.0), (T - window - 1, 6.0)):
                if 0 <= at < T:
                    self.rows[i][at, R:] = (size * last[d:]).to(dtype)
                    self.rows[i][at, :R] = size
        self.want = []
        for i, T in enumerate(lens):
            c, kr = self.rows[i][:, :R].double(), self.rows[i][:, R:].double()
            k = torch.cat([torch.einsum("tr,hdr->thd", c, self.uk.double()), kr[:, None].expand(-1, H, -1)], -1)
            v = torch.einsum("tr,hnr->thn", c, self.uv.double())
            self.want.append(O.attend(self.q[i].double(), k, v, self.s.scale, O.window_mask(T, window),
                                      None if self.sinks is None else self.sinks.double()))
        self.cache = self.c.pool(1, self.s.row, [x.float()[:, None] for x in self.rows], dtype)
        self.cache[..., R + r:] = 0                          # the padding of written rows is zero

    def to(self, x):
        return None if x is None else x.to(self.device)

    def folded(self, news, **kw):
        """Through the queries folded into latents."""
        s = self.s
        x = torch.cat([q[-m:] for q, m in zip(self.q, news)]).to(self.device)
        q = torch.zeros(s.heads, x.shape[0], s.row, dtype=self.dtype, device=self.device)
        q[..., s.rank:s.rank + s.rot] = x[..., s.dim:].transpose(0, 1)
        ops.head_linear(x[..., :s.dim].transpose(0, 1).contiguous(), self.to(self.uk).transpose(1, 2).contiguous(), out=q[..., :s.rank])
        run = lambda a, b, e, m: ops.latent_attention(s, q, self.cache, self.to(self.c.table), e, q_start=a, q_lens=b,
                                                      sinks=self.to(self.sinks), **kw)
        o = attend_all(self.c, news, run)
        return ops.head_linear(o, self.to(self.uv)).transpose(0, 1)

    def decode(self, **kw):
        s = self.s
        x = torch.stack([q[-1] for q in self.q]).to(self.device)
        q = torch.zeros(s.heads, x.shape[0], s.row, dtype=self.dtype, device=self.device)
        q[..., s.rank:s.rank + s.rot] = x[..., s.dim:].transpose(0, 1)
        ops.head_linear(x[..., :s.dim].transpose(0, 1).contiguous(), self.to(self.uk).transpose(1, 2).contiguous(), out=q[..., :s.rank])
        o = ops.latent_attention(s, q, self.cache, self.to(self.c.table), i32(self.lens, self.device), sinks=self.to(self.sinks), **kw)
        return ops.head_linear(o, self.to(self.uv)).transpose(0, 1)

    def expanded(self, news):
        """Through keys and values of the pages the new tokens see."""
        s, (nk, _) = self.s, self.s.slabs
        x = torch.cat([q[-m:] for q, m in zip(self.q, news)])
        q = torch.zeros(x.shape[0], s.heads, 64 * nk, dtype=self.dtype)
        q[..., :s.dim] = x[..., :s.dim]
        q[..., 64 * nk - 64:64 * nk - 64 + s.rot] = x[..., s.dim:]
        pages, base, at = [], [], 0
        for b, (T, m) in enumerate(zip(self.lens, news)):
            lo = max(0, T - m - s.window + 1) // 32
            pages += self.c.table[b, lo:self.c.pages[b]].tolist()
            base.append((at - lo) * 32)
            at += self.c.pages[b] - lo
        lat, r = ops.latent_gather(s, self.cache, i32(pages, self.device), (s.rot + 7) // 8 * 8)
        w = torch.cat([self.uk.reshape(-1, s.rank), self.uv.reshape(-1, s.rank)]).to(self.device)
        kv = ops.linear(lat, w, swap=False)
        return attend_all(self.c, news, lambda a, b, e, m: ops.latent_prefill(s, q.to(self.device), kv, r, i32(base, self.device), a, b, e,
                                                                              m, self.to(self.sinks)))

    def last(self, news):
        return torch.cat([w[-m:] for w, m in zip(self.want, news)])


@on_devices
@in_dtypes
@pytest.mark.parametrize("sizes", LATENT)
@pytest.mark.parametrize("window", [1, 30, 33, 130, 1000])
def test_latent_attention(device, dtype, sizes, window):
    lens = [200, 33, 98]
    x = Latent(sizes, dtype, device, lens, window)
    tol = TOL[dtype] if dtype == torch.float32 else 3e-2
    for news in ([7, 33, 1], [60, 2, 98]):
        close(x.folded(news), x.last(news), tol, f"folded {news}")
    for splits in (1, 2, 4, 8):
        close(x.decode(num_splits=splits), torch.stack([w[-1] for w in x.want]), tol, f"decode, {splits} splits")
        close(x.folded([3, 3, 3], num_splits=splits), x.last([3, 3, 3]), tol, f"three tokens, {splits} splits")
    if x.s.slabs is not None and dtype == torch.bfloat16:
        for news in (lens, [60, 33, 2], [1, 2, 98], [140, 1, 1]):
            close(x.expanded(news), x.last(news), tol, f"expanded {news}")


@on_devices
def test_a_sink_takes_its_share_once(device):
    """A sink as large as the only visible score halves the result; without one the value comes through whole."""
    sizes = LATENT[0]
    for dtype in (torch.float32, torch.bfloat16):
        x = Latent(sizes, dtype, device, [40, 1], 1, sinks=False)
        whole = torch.stack([w[-1] for w in x.want])
        close(x.decode(), whole, 2e-2)
        H, d, r, n, R, Q = sizes
        c, kr = x.rows[0][-1, :R].double(), x.rows[0][-1, R:].double()
        q = x.q[0][-1].double()
        score = (torch.einsum("hd,hdr,r->h", q[:, :d], x.uk.double(), c) + q[:, d:] @ kr) * x.s.scale
        x.sinks = score.float()
        close(x.decode()[0], whole[0] / 2, 2e-2)


@on_devices
def test_rows_without_a_sequence_stay_out(device):
    """Decode rows with a negative length write zeros and disturb no other row."""
    for dtype in (torch.float32, torch.bfloat16):
        x = Latent(LATENT[0], dtype, device, [70, 40, 33], 50)
        x.lens = [70, -1, 33]
        for splits in (1, 2):
            got = x.decode(num_splits=splits)
            close(got[0], x.want[0][-1], 3e-2)
            close(got[2], x.want[2][-1], 3e-2)
            assert (got[1] == 0).all()


@pytest.mark.gpu
@pytest.mark.parametrize("heads", [16, 32, 40])
def test_long_contexts_on_the_tensor_cores(heads):
    """Thousands of tokens: rings of pages wrap many times, in every split."""
    x = Latent((heads, 32, 64, 40, 512, 40), torch.bfloat16, "cuda", [2500, 1, 700], 2100)
    for splits in (1, 4, 8):
        close(x.decode(num_splits=splits), torch.stack([w[-1] for w in x.want]), 3e-2, f"{splits} splits")
    assert math.isfinite(x.want[0].sum())
