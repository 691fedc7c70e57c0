"""Each mechanism of the pre-norm layer-by-layer decoders against the plain statement in mumilorn_oracle.py: the operators'
PyTorch form on the CPU and the kernels on a GPU, in 32-bit and in bfloat16."""
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import mumilorn_oracle as O  # noqa: E402

from nkipy_b200 import ops  # noqa: E402
from nkipy_b200.ops import Branch, Decay, MapsSpec, Proj  # noqa: E402
from nkipy_b200.ops.linear_attention import linear_state_shape  # noqa: E402

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


# --------------------------------------------------------------------------- residual branches, activations
@on_devices
@in_dtypes
@pytest.mark.parametrize("form", ["f32", "bf16", "partials"])
@pytest.mark.parametrize("width", [96, 70, 2048])
def test_scaled_and_routed_branches_of_a_residual_update(device, dtype, form, width):
    T, k, eps = 5, 3, 1e-4
    x, w = rnd(T, width, seed=1), rnd(width, seed=2)
    y, yv = projection(rnd(T, width + 4, seed=3), form)
    rows, rv = projection(rnd(T * k, width, seed=4), "bf16" if form == "bf16" else "f32")
    pos = torch.randperm(T * k, generator=torch.Generator().manual_seed(5)).to(torch.int32)
    pos[4] = -1                                             # a pair that is handled elsewhere
    pw = rnd(T, k, seed=6)
    d = lambda t: t.to(device)
    want = x.double() + 0.7 * yv[:, 4:]
    routed = torch.zeros(T, width, dtype=torch.float64)
    for t in range(T):
        for j in range(k):
            if pos[t * k + j] >= 0:
                routed[t] += pw[t, j].double() * rv[pos[t * k + j].long()]
    branches = [Branch(Proj(d(y), 4, width), scale=0.7), Branch(Proj(d(rows), 0, width), scale=1.5, pair_pos=d(pos), pair_w=d(pw))]
    for n, wanted in ((1, want), (2, want + 1.5 * routed)):
        r, (h,) = ops.gated_residual(d(x), branches[:n], norms=[d(1 + w)], eps=eps, dtype=dtype)
        close(r, wanted, 1e-5, "residual")
        close(h, O.pre_norm(wanted, w.double(), eps), TOL[dtype], "norm")
    r, _ = ops.gated_residual(d(x), branches[1:])
    close(r, x.double() + 1.5 * routed, 1e-5, "routed alone")


@on_devices
@in_dtypes
@pytest.mark.parametrize("form", ["f32", "bf16", "partials"])
@pytest.mark.parametrize("n", [24, 31])
def test_single_activations(device, dtype, form, n):
    y, v = projection(rnd(6, n + 9, std=2.0), form)
    v = v[:, 8:8 + n]
    for act, want in (("relu2", torch.relu(v) ** 2), ("tanh", torch.tanh(v)), ("sigmoid", torch.sigmoid(v)), ("silu", O.silu(v)),
                      ("none", v)):
        close(ops.activation(Proj(y.to(device), 8, n), act, dtype=dtype), want, TOL[dtype], act)


@on_devices
@pytest.mark.parametrize("tokens,n", [(130, 96), (200, 384), (600, 384), (140, 33)])
def test_squared_relu_in_the_gemm_epilogue(device, tokens, n):
    x, w = rnd(tokens, 128).bfloat16(), rnd(n, 128, seed=1, std=0.2).bfloat16()
    got = ops.linear(x.to(device), w.to(device), swap=False, out_act="relu2")
    close(got, torch.relu(x.double() @ w.double().T) ** 2, 1e-2)


# --------------------------------------------------------------------------- token mix
@on_devices
@in_dtypes
@pytest.mark.parametrize("width,lens", [(40, [7, 1, 2, 30]), (33, [5, 19]), (1100, [9, 1, 1]), (24, [600, 3, 17])])
def test_token_mix_whole_portions_and_single_tokens(device, dtype, width, lens):
    mu = torch.rand(5, width, generator=torch.Generator().manual_seed(3))
    h = [rnd(n, width, seed=10 + i).to(dtype) for i, n in enumerate(lens)]
    want = [torch.stack([O.token_mix(x.double(), m.double()) for m in mu]) for x in h]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)
    slots = list(range(len(lens), 0, -1))                       # slot 0 stays free
    state = torch.full((len(lens) + 1, width), 9.0, device=device)

    def run(parts):
        """parts: (sequence, first, end)"""
        q_lens = [e - f for _, f, e in parts]
        starts = [sum(q_lens[:i]) for i in range(len(parts))]
        x = torch.cat([h[b][f:e] for b, f, e in parts]).to(device)
        out = ops.token_mix(x, mu.to(device), state, i32([e for _, _, e in parts]), q_start=i32(starts), q_lens=i32(q_lens),
                            rows=i32([slots[b] for b, _, _ in parts]))
        close(out, torch.cat([want[b][:, f:e] for b, f, e in parts], 1), TOL[dtype])

    run([(b, 0, n) for b, n in enumerate(lens)])
    for first in (1, 2):                                        # the slots hold other sequences' rows now
        run([(b, 0, min(first, n)) for b, n in enumerate(lens)])
        rest = [(b, first, min(first + 2, n)) for b, n in enumerate(lens) if n > first]
        run(rest)
        more = [(b, first + 2, n) for b, n in enumerate(lens) if n > first + 2]
        if more:
            run(more)
    assert (state[0] == 9).all()
    # a decode step, one row inactive: its slot keeps its row
    B = len(lens)
    state = torch.stack([x[-1].float() for x in h]).to(device)
    new = rnd(B, width, seed=99).to(dtype)
    ctx = [n + 1 for n in lens]
    ctx[-1] = -1
    out = ops.token_mix(new.to(device), mu.to(device), state, i32(ctx))
    for b in range(B - 1):
        full = torch.cat([h[b], new[b:b + 1]]).double()
        close(out[:, b], torch.stack([O.token_mix(full, m.double())[-1] for m in mu]), TOL[dtype], f"step {b}")
        assert torch.equal(state[b].cpu(), new[b].float())
    assert torch.equal(state[-1].cpu(), h[-1][-1].float())


# --------------------------------------------------------------------------- decays and recurrences
@on_devices
@in_dtypes
@pytest.mark.parametrize("tokens,rank,n", [(3, 16, 70), (40, 5, 64), (150, 16, 96), (150, 12, 33), (1, 70, 128)])
def test_low_rank_products(device, dtype, tokens, rank, n):
    x, xv = projection(rnd(tokens, rank + 8), "bf16" if dtype == torch.bfloat16 else "partials")
    w = rnd(n, rank, seed=1).to(dtype)
    for act, f in (("none", lambda z: z), ("tanh", torch.tanh)):
        got = ops.low_rank(Proj(x.to(device), 8, rank), w.to(device), act)
        assert got.dtype == torch.float32
        close(got, f(xv[:, 8:]) @ w.double().T, 2e-5 if dtype == torch.float32 or tokens <= 128 else 1e-2)


class Recurrence:
    """Projections of one sequence and everything around the state of its heads."""

    def __init__(self, T, H, d, n, kind, dtype, seed=0, rank=6, tau=3.0, shared=None):
        self.T, self.H, self.d, self.n, self.kind, self.dtype, self.tau, self.rank = T, H, d, n, kind, dtype, tau, rank
        form = "bf16" if dtype == torch.bfloat16 else "f32"
        self.widths = [H * d, H * d, H * n, H * n, rank]
        self.z, self.zv = projection(rnd(T, sum(self.widths), seed=seed), form)
        c = shared or self
        if shared is None:
            self.w = rnd(H * d, rank, seed=seed + 1, std=0.5).to(dtype)
            self.bias = rnd(H * d, seed=seed + 2) + (1.0 if kind == "sigmoid_root" else -2.0)
            self.bonus = 1.5 * rnd(H * d, seed=seed + 3) if kind == "double_exp" else None
            self.norm = 1 + 0.3 * rnd(n if kind == "sigmoid_root" else H * n, seed=seed + 4)
        else:
            self.w, self.bias, self.bonus, self.norm = c.w, c.bias, c.bonus, c.norm
        self.act = "none" if kind == "sigmoid_root" else "tanh"

    def want(self, eps=1e-5, q_scale=0.5, scale=0.8):
        T, H, d, n = self.T, self.H, self.d, self.n
        q, k, v, g, x = self.zv.split(self.widths, 1)
        x = torch.tanh(x) if self.act == "tanh" else x
        z = x @ self.w.double().T + self.bias.double()
        q, k, v = (q * q_scale).view(T, H, d), k.view(T, H, d), v.view(T, H, n)
        if self.kind == "sigmoid_root":
            o = O.linear_attention(q, k, v, O.sigmoid_root_decay(z, self.tau).view(T, H, d))
        else:
            o = O.bonus_attention(q, k, v, O.double_exp_decay(z).view(T, H, d), self.bonus.double().view(H, d))
        o = O.rms(o, eps) * self.norm.double().view(-1, n)
        return scale * o.reshape(T, -1) * O.silu(g)

    def slices(self, z):
        out, c = [], 0
        for w in self.widths:
            out.append(Proj(z, c, w))
            c += w
        return out

    def run(self, z, state, ctx, out=None, **kw):
        dev = state.device
        q, k, v, g, x = self.slices(z)
        decay = Decay(self.kind, x, self.w.to(dev), self.bias.to(dev), self.act, self.tau)
        return ops.linear_attention(q, k, v, decay, g, self.norm.to(dev), state, ctx, heads=self.H, dim=self.d, vdim=self.n,
                                    eps=1e-5, q_scale=0.5, scale=0.8, bonus=None if self.bonus is None else self.bonus.to(dev),
                                    dtype=self.dtype, out=out, **kw)


kinds = pytest.mark.parametrize("kind", ["sigmoid_root", "double_exp"])
I32 = lambda x, device: torch.tensor(x, dtype=torch.int32, device=device)


@on_devices
@in_dtypes
@kinds
@pytest.mark.parametrize("H,d,n", [(2, 44, 56), (3, 20, 28), (1, 128, 128), (2, 7, 5), (2, 160, 40), (1, 64, 200), (1, 1, 1)])
def test_recurrence_whole_portions_and_single_tokens_agree(device, dtype, kind, H, d, n):
    c = Recurrence(45, H, d, n, kind, dtype)
    want = c.want()

    def feed(cuts, steps_from=None):
        state = torch.full((3, *linear_state_shape(H, d, n)), 7.0, device=device)      # slots that were used before
        outs, lo = [], 0
        for m in cuts:
            z = c.z[lo:lo + m].to(device)
            kw = dict(rows=I32([1], device))
            if steps_from is None or lo < steps_from:
                kw.update(q_start=I32([0], device), q_lens=I32([m], device))
            outs.append(c.run(z, state, I32([lo + m], device), **kw))
            lo += m
        assert (state[0] == 7).all() and (state[2] == 7).all()
        return torch.cat(outs)

    for cuts in ([45], [1] * 3 + [2] * 4 + [16, 1, 17], [31, 2, 12], [8, 8, 29]):
        close(feed(cuts), want, TOL[dtype], f"cuts {cuts}")
    close(feed([30] + [1] * 15, steps_from=1), want, TOL[dtype], "prompt, then single tokens")
    close(feed([1] * 45, steps_from=0), want, TOL[dtype], "single tokens")


@on_devices
@in_dtypes
@kinds
def test_recurrence_over_many_sequences_and_wide_grids(device, dtype, kind):
    """Enough CTAs for every column width of the scan, a batch beyond 128 tokens, results into a slice of columns."""
    H, d, n = 4, 64, 64
    for B in (1, 20, 80):
        lens = [3 + (7 * b) % 29 for b in range(B)]
        first = Recurrence(lens[0], H, d, n, kind, dtype)
        cs = [first] + [Recurrence(m, H, d, n, kind, dtype, seed=50 * b, shared=first) for b, m in enumerate(lens) if b > 0]
        z = torch.cat([c.z for c in cs]).to(device)
        starts = [sum(lens[:b]) for b in range(B)]
        slots = torch.randperm(B + 1, generator=torch.Generator().manual_seed(1))[:B].tolist()
        state = torch.full((B + 1, *linear_state_shape(H, d, n)), 3.0, device=device)
        out = torch.full((sum(lens), H * n + 5), 2.0, dtype=dtype, device=device)
        first.run(z, state, I32(lens, device), out=out[:, 5:], q_start=I32(starts, device), q_lens=I32(lens, device),
                  rows=I32(slots, device))
        close(out[:, 5:], torch.cat([c.want() for c in cs]), TOL[dtype], f"batch {B}")
        assert (out[:, :5] == 2).all()


@on_devices
@kinds
def test_recurrence_reads_partial_sums_and_skips_inactive_rows(device, kind):
    H, d, n = 2, 24, 36
    cs = [Recurrence(9, H, d, n, kind, torch.float32, seed=3)]
    cs.append(Recurrence(14, H, d, n, kind, torch.float32, seed=77, shared=cs[0]))
    state = torch.zeros((4, *linear_state_shape(H, d, n)), device=device)
    part = lambda z: torch.stack([z - 1.0, torch.ones_like(z)]).to(device)
    z = torch.cat([cs[0].z[:8], cs[1].z[:13]])
    cs[0].run(part(z), state, I32([8, 13], device), q_start=I32([0, 8], device), q_lens=I32([8, 13], device),
              rows=I32([2, 0], device))
    before = state.clone()
    step = torch.zeros(4, z.shape[1])
    step[2], step[0] = cs[0].z[8], cs[1].z[13]
    out = cs[0].run(part(step), state, I32([14, -1, 9, -1], device))
    close(out[2], cs[0].want()[-1], 2e-5)
    close(out[0], cs[1].want()[-1], 2e-5)
    assert torch.equal(state[[1, 3]], before[[1, 3]]) and (out[[1, 3]] == 0).all()


@on_devices
@kinds
def test_decays_at_their_extremes(device, kind):
    """Channels that keep everything, forget at once, and logits far out on both sides."""
    T, H, d, n = 40, 1, 8, 8
    c = Recurrence(T, H, d, n, kind, torch.float32, tau=2.0)
    c.w = torch.zeros_like(c.w)
    c.bias = torch.tensor([40.0, -40.0, 90.0, -90.0, 0.0, 5.0, -5.0, 1.0])
    state = torch.zeros((1, *linear_state_shape(H, d, n)), device=device)
    kw = dict(q_start=I32([0], device), q_lens=I32([T], device))
    close(c.run(c.z.to(device), state, I32([T], device), **kw), c.want(), 2e-5)
    assert torch.isfinite(state).all()


@on_devices
@kinds
def test_a_write_survives_hundreds_of_tokens(device, kind):
    """One channel hardly forgets and carries the first token's value to the end; the others see noise only."""
    T, d, n = 400, 32, 32
    c = Recurrence(T, 1, d, n, kind, torch.float32, tau=8.0)
    z = 0.05 * c.zv.float()
    q, k, v, g, x = z.split(c.widths, 1)
    k[0, 5], v[0], q[-1] = 30.0, 10 * rnd(n, seed=3), 0.0
    q[-1, 5], g[-1] = 6.0, 1.0
    k[1:, 5] = 0.0
    c.z, c.zv = z, z.double()
    c.bias = torch.full((d,), 0.5)
    c.bias[5] = 12.0 if kind == "sigmoid_root" else -9.0
    c.norm = torch.ones_like(c.norm)
    want = c.want()[-1]
    assert torch.nn.functional.cosine_similarity(want, v[0].double(), dim=0) > 0.99
    state = torch.zeros((1, *linear_state_shape(1, d, n)), device=device)
    for lo, hi in ((0, 2), (2, 300), (300, T)):
        out = c.run(z[lo:hi].to(device), state, I32([hi], device), q_start=I32([0], device), q_lens=I32([hi - lo], device))
    close(out[-1], want, 1e-4)


@on_devices
@in_dtypes
@pytest.mark.parametrize("H,n,pad", [(3, 40, 24), (2, 64, 64), (5, 7, 1), (2, 200, 0)])
def test_gates_of_heads(device, dtype, H, n, pad):
    T = 6
    x = rnd(T, H, n + pad, seed=1).to(dtype)
    g, gv = projection(rnd(T, H * n + 4, seed=2), "partials" if dtype == torch.float32 else "bf16")
    gate = Proj(g.to(device), 4, H * n)
    gv, xv, hv = gv[:, 4:], x[:, :, :n].double(), x.to(device)[:, :, :n]
    got = ops.gate_heads(hv, gate, "sigmoid", scale=0.6)
    close(got, 0.6 * xv.reshape(T, -1) * torch.sigmoid(gv), TOL[dtype], "sigmoid")
    out = torch.full((T, H * n + 3), 4.0, dtype=dtype, device=device)
    for w in (1 + rnd(n, seed=3), 1 + rnd(H * n, seed=4)):
        ops.gate_heads(hv, gate, "silu", norm_w=w.to(device), eps=1e-3, out=out[:, 3:])
        close(out[:, 3:], (O.rms(xv, 1e-3) * w.double().view(-1, n)).reshape(T, -1) * O.silu(gv), TOL[dtype], "silu, normed")
    assert (out[:, :3] == 4).all()


# --------------------------------------------------------------------------- attention
@on_devices
@in_dtypes
@pytest.mark.parametrize("form", ["f32", "bf16", "partials"])
@pytest.mark.parametrize("H,G,d,v", [(4, 2, 24, 40), (3, 3, 64, 64), (6, 1, 12, 9), (2, 1, 100, 128)])
def test_query_and_key_norms_over_all_heads(device, dtype, form, H, G, d, v):
    T, eps = 70, 1e-3
    spec = MapsSpec(H, G, d, v, 1.0, maps=1, eps=eps, tiled=dtype == torch.bfloat16)
    z = rnd(T, d * (H + G) + v * G)
    z[:, :d] *= 30                                            # one head much larger: a norm per head would show
    zt, zv = projection(z, form)
    qn, kn = 1 + rnd(H * d, seed=1), 1 + rnd(G * d, seed=2)
    kc = torch.zeros((4, G, 32, spec.dim_p), dtype=dtype, device=device)
    vc = torch.zeros((4, G, 32, spec.vdim_p), dtype=dtype, device=device)
    order = torch.randperm(4 * 32, generator=torch.Generator().manual_seed(1))[:T].to(torch.int32)
    order[7] = -1                                             # a token that is not stored
    zz = zt.to(device)
    q = ops.row_norm_append(spec, Proj(zz, 0, H * d), Proj(zz, H * d, G * d), Proj(zz, (H + G) * d, G * v), qn.to(device),
                            kn.to(device), order.to(device), kc, vc)
    tol = TOL[dtype] if dtype == torch.bfloat16 else 2e-6
    close(q[..., :d].reshape(T, -1), O.row_norm(zv[:, :H * d], qn.double(), eps), tol, "queries")
    assert (q[..., d:] == 0).all() and (kc[..., d:] == 0).all() and (vc[..., v:] == 0).all()
    keep = order >= 0
    at = lambda c: c.cpu()[(order // 32).long(), :, (order % 32).long()][keep]
    close(at(kc)[..., :d].reshape(-1, G * d), O.row_norm(zv[:, H * d:(H + G) * d], kn.double(), eps)[keep], tol, "keys")
    close(at(vc)[..., :v].reshape(-1, G * v), zv[keep, (H + G) * d:], tol, "values")


class WindowCase:
    """Queries, keys and values of several sequences in a paged cache with scattered blocks."""

    def __init__(self, lens, H, G, d, v, window, device, dtype, std=1.0, seed=0):
        self.spec = MapsSpec(H, G, d, v, d ** -0.5, maps=1, window=window, tiled=dtype == torch.bfloat16)
        self.device, self.dtype, self.lens = device, dtype, lens
        self.q = [rnd(n, H, d, seed=seed + 3 * i, std=std).to(dtype) for i, n in enumerate(lens)]
        self.k = [rnd(n, G, d, seed=seed + 3 * i + 1, std=std).to(dtype) for i, n in enumerate(lens)]
        self.v = [rnd(n, G, v, seed=seed + 3 * i + 2).to(dtype) for i, n in enumerate(lens)]

    def fill(self):
        s = self.spec
        pages = [(n + 31) // 32 for n in self.lens]
        total = sum(pages) + 3
        perm = torch.randperm(total, generator=torch.Generator().manual_seed(9)).tolist()
        kc, vc = torch.zeros((total, s.kv_heads, 32, s.dim_p)), torch.zeros((total, s.kv_heads, 32, s.vdim_p))
        kc[..., :s.dim], vc[..., :s.vdim] = 9.0, -50.0        # pages hold values of earlier owners
        self.table = torch.zeros((len(self.lens), max(pages) + 2), dtype=torch.int32)
        for b, n in enumerate(self.lens):
            for j in range(pages[b]):
                blk = perm.pop()
                self.table[b, j] = blk
                m = min(32, n - 32 * j)
                kc[blk, :, :m, :s.dim] = self.k[b][32 * j:32 * j + m].float().transpose(0, 1)
                vc[blk, :, :m, :s.vdim] = self.v[b][32 * j:32 * j + m].float().transpose(0, 1)
        self.kc, self.vc = kc.to(self.device, self.dtype), vc.to(self.device, self.dtype)
        return self

    def want(self, b):
        s = self.spec
        n = self.lens[b]
        mask = O.window_mask(n, s.window or n + 1)
        return O.softmax_attention(self.q[b].double(), self.k[b].double(), self.v[b].double(), s.scale, mask)

    def run(self, parts, step=False):
        """parts: (sequence, first, end) of the new tokens; step: the decode form."""
        s = self.spec
        q = torch.zeros((sum(e - f for _, f, e in parts), s.heads, s.dim_p))
        o, starts = 0, []
        for b, f, e in parts:
            starts.append(o)
            q[o:o + e - f, :, :s.dim] = self.q[b][f:e].float()
            o += e - f
        q, rows = q.to(self.device, self.dtype), [b for b, _, _ in parts]
        i32 = lambda x: I32(x, self.device)
        kw = {} if step else dict(q_start=i32(starts), q_lens=i32([e - f for _, f, e in parts]),
                                  max_q_len=max(e - f for _, f, e in parts))
        return ops.heads_attention(s, q, self.kc, self.vc, self.table[rows].to(self.device), i32([e for _, _, e in parts]), **kw)


SIZES = [(6, 3, 28, 64), (4, 4, 24, 40), (6, 1, 64, 128), (2, 1, 48, 80), (20, 1, 16, 128), (2, 2, 144, 72)]


@on_devices
@in_dtypes
@pytest.mark.parametrize("window", [0, 1, 45, 300])
@pytest.mark.parametrize("H,G,d,v", SIZES)
def test_windowed_attention_in_prompts_and_single_tokens(device, dtype, window, H, G, d, v):
    lens = [1, 33, 150, 290]
    c = WindowCase(lens, H, G, d, v, window, device, dtype, std=1.3).fill()
    want = [c.want(b) for b in range(len(lens))]
    close(c.run([(b, 0, n) for b, n in enumerate(lens)]), torch.cat(want), TOL[dtype], "whole prompts")
    parts = [(2, 31, 33), (3, 100, 289), (1, 32, 33), (0, 0, 1)]
    close(c.run(parts), torch.cat([want[b][f:e] for b, f, e in parts]), TOL[dtype], "portions")
    for back in (1, 2, 20, 33):
        rows = [(b, n - back, n - back + 1) for b, n in enumerate(lens) if n >= back]
        close(c.run(rows, step=True), torch.stack([want[b][f] for b, f, _ in rows]), TOL[dtype], f"{back} from the end")


@on_devices
@in_dtypes
@pytest.mark.parametrize("window", [2, 31, 32, 33, 64, 128, 129])
def test_a_key_just_inside_and_just_outside_the_window(device, dtype, window):
    """One key fits every query and takes nearly all the weight as long as it is visible: the last query that sees it and the
    first that does not are told apart, wherever pages and tiles end."""
    n, d, v = 290, 32, 64
    for key in (0, 31, 32, 127, 128, 150):
        c = WindowCase([n], 2, 1, d, v, window, device, dtype, std=0.3)
        target = rnd(d, seed=42)
        target = (8 * target / target.norm()).to(dtype)
        c.k[0][key, 0] = target
        c.q[0][:] = target * 1.5
        c.fill()
        want = c.want(0)
        inside, outside = key + window - 1, key + window
        cos = lambda x: torch.nn.functional.cosine_similarity(x[0].double(), c.v[0][key, 0].double(), dim=0)
        if outside >= n:
            continue
        assert cos(want[inside]) > 0.9 > 0.6 > cos(want[outside])
        close(c.run([(0, 0, n)]), want, TOL[dtype], "prompt")
        close(c.run([(0, inside, inside + 2)]), want[inside:inside + 2], TOL[dtype], "portion over the edge")
        for pos in (inside, outside):
            close(c.run([(0, pos, pos + 1)], step=True), want[pos:pos + 1], TOL[dtype], "single token")


@on_devices
@in_dtypes
def test_inactive_rows_of_a_windowed_step_write_zeros(device, dtype):
    for heads in (6, 40):                                       # also more query heads per key head than a fragment holds
        c = WindowCase([40, 70], heads, 2, 32, 64, 17, device, dtype).fill()
        q = torch.zeros((3, heads, c.spec.dim_p), dtype=dtype)
        q[1, :, :32] = c.q[1][69]
        table = torch.stack([c.table[0], c.table[1], c.table[0]]).to(device)
        out = ops.heads_attention(c.spec, q.to(device), c.kc, c.vc, table, I32([-1, 70, -1], device))
        close(out[1], c.want(1)[69], TOL[dtype])
        assert (out[[0, 2]] == 0).all()


# --------------------------------------------------------------------------- routed experts
@on_devices
@pytest.mark.parametrize("form", ["f32", "partials"])
@pytest.mark.parametrize("E,top,groups,keep", [(8, 3, 4, 2), (6, 2, 2, 1), (6, 6, 3, 3), (12, 1, 12, 5), (40, 4, 5, 2), (64, 8, 2, 2),
                                               (9, 4, 0, 0)])
def test_router_with_groups(device, form, E, top, groups, keep):
    T = 50
    z, zv = projection(rnd(T, E, std=2.0), form)
    w, e = ops.router_topk(z.to(device), top, groups=groups, keep=keep, scale=2.5)
    limited = 0
    for t in range(T):
        pick, weight = O.route(zv[t], top, dict(count=groups, keep=keep) if groups else None, 2.5)
        assert e[t].tolist() == pick
        close(w[t], weight, 1e-5)
        limited += sorted(pick) != sorted(zv[t].topk(top).indices.tolist())
    assert limited > 0 or keep == groups or top == 1            # the groups do exclude an expert somewhere


@on_devices
@in_dtypes
@pytest.mark.parametrize("W,ff,E,top,tokens", [(64, 40, 6, 2, 50), (96, 64, 4, 4, 1), (64, 24, 8, 3, 3000), (30, 7, 5, 2, 9)])
def test_routed_experts(device, dtype, W, ff, E, top, tokens):
    from nkipy_b200.models.config import ExpertsSpec
    from nkipy_b200.models.mixers import Tensors
    from nkipy_b200.models.moe import RoutedExperts

    ws = {"router": rnd(E, W, seed=1, std=4 / W ** 0.5)}
    for e in range(E):
        for i, n in enumerate(("gate", "up", "down")):
            ws[f"e{e}.{n}"] = rnd(*((W, ff) if n == "down" else (ff, W)), seed=10 * e + i + 2, std=W ** -0.5)
    ws = {k: v.bfloat16() for k, v in ws.items()}
    spec = ExpertsSpec(E, top, ff, 0, 0, 1.4)
    block = RoutedExperts(spec, Tensors(lambda k: ws[k].to(device), "", dtype))
    h = rnd(tokens, W, seed=99).to(dtype)
    got = ops.gated_residual(torch.zeros(tokens, W, device=device), block.run(None, h.to(device)))[0].cpu()
    some = range(tokens) if tokens < 100 else range(0, tokens, 97)
    m = {"router": {"top": top, "groups": None, "scale": 1.4}}
    want = O.experts(h[list(some)].double(), {k: v.double() for k, v in ws.items()}, m)
    close(got[list(some)], want, TOL[dtype])
