"""Each mechanism of the layer-by-layer decoders against the plain statement in hybrid_oracle.py: the operators' PyTorch
form on the CPU and the kernels on a GPU, in 32-bit and in bfloat16."""
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import hybrid_oracle as O  # noqa: E402

from nkipy_b200 import ops  # noqa: E402
from nkipy_b200.models import config as C  # noqa: E402
from nkipy_b200.ops import MapsSpec, Proj  # noqa: E402
from nkipy_b200.ops.mixers import hgrn2_state_shape  # noqa: E402

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
on_devices = pytest.mark.parametrize("device", DEVICES)
in_dtypes = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}


@pytest.fixture(autouse=True, scope="module")
def _one_thread():
    """The small tensors of these tests gain nothing from threads and lose a lot when several test processes share cores."""
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


# --------------------------------------------------------------------------- residual, norms, gates
@on_devices
@in_dtypes
@pytest.mark.parametrize("form", ["f32", "bf16", "partials"])
@pytest.mark.parametrize("width,groups", [(96, 3), (70, 7), (2048, 4), (48, 48), (520, 1)])
def test_gated_residual_and_group_norms(device, dtype, form, width, groups):
    T, eps = 5, 1e-3
    x = rnd(T, width, seed=1)
    x[:, : width // groups] *= 50                      # groups of very different size: a norm over all would show
    mk = lambda seed: projection(rnd(T, 3 * width + 6, seed=seed), form)
    (y1, y1v), (y2, y2v) = mk(2), mk(3)
    b1, b2, row, mat = rnd(width, seed=7), rnd(width, seed=8), rnd(width, seed=9), rnd(T, width, seed=10)
    w1, w2 = 1 + rnd(width, seed=11), 1 + rnd(width, seed=12)
    d = lambda t: t.to(device)
    branches = [(Proj(d(y1), 0, width), Proj(d(y1), width + 2, width), d(b1)),
                (Proj(d(y2), 2 * width + 6, width), Proj(d(y2), width, width), d(b2))]
    sl = lambda v, c: v[:, c:c + width]
    base = x.double()
    for n in (0, 1, 2):
        want = base
        if n > 0:
            want = want + sl(y1v, 0) * torch.sigmoid(sl(y1v, width + 2) + b1.double())
        if n > 1:
            want = want + sl(y2v, 2 * width + 6) * torch.sigmoid(sl(y2v, width) + b2.double())
        want = want + mat.double() + row.double()
        r, (h1, h2) = ops.gated_residual(d(x), branches[:n], add_mat=d(mat), add_row=d(row), norms=[d(w1), d(w2)],
                                         groups=groups, eps=eps, dtype=dtype)
        close(r, want, 1e-5, "residual")
        assert h1.dtype == dtype
        close(h1, O.group_norm(want, w1.double(), groups, eps), TOL[dtype], "norm 1")
        close(h2, O.group_norm(want, w2.double(), groups, eps), TOL[dtype], "norm 2")


@on_devices
@in_dtypes
def test_embedding_is_scaled_in_32_bit(device, dtype):
    table = rnd(20, 72).to(dtype)
    ids = torch.tensor([3, 19, 0, 3], dtype=torch.int32)
    x, hs = ops.gated_residual(None, ids=ids.to(device), table=table.to(device), scale=3.7, dtype=dtype)
    assert x.dtype == torch.float32 and hs == []
    close(x, O.embed(table.double(), ids.long(), 3.7), 1e-6)


@on_devices
@in_dtypes
@pytest.mark.parametrize("form", ["f32", "bf16", "partials"])
@pytest.mark.parametrize("inter", [24, 31])
def test_gated_activation(device, dtype, form, inter):
    y, v = projection(rnd(6, 2 * inter + 9, std=3.0), form)
    p = lambda c: Proj(y.to(device), c, inter)
    got = ops.gated_act(p(0), p(inter), "gelu_tanh", dtype=dtype)
    close(got, O.gelu_tanh(v[:, :inter]) * v[:, inter:2 * inter], TOL[dtype])
    got = ops.gated_act(p(0), p(inter), "silu", dtype=dtype)
    close(got, v[:, :inter] * torch.sigmoid(v[:, :inter]) * v[:, inter:2 * inter], TOL[dtype])


@on_devices
@pytest.mark.parametrize("tokens", [1, 40, 200, 600])
def test_gelu_in_the_gemm_epilogue(device, tokens):
    x, w = rnd(tokens, 128).bfloat16(), rnd(2 * 384, 128, seed=1, std=0.2).bfloat16()
    got = ops.linear(x.to(device), w.to(device), gated=True, act="gelu_tanh", swap=False if tokens > 128 else None)
    g, u = x.double() @ w[:384].double().T, x.double() @ w[384:].double().T
    close(got, O.gelu_tanh(g) * u, 1e-2)


@on_devices
@pytest.mark.parametrize("m,n,k", [(1, 5, 7), (70, 130, 33), (64, 64, 64), (3, 300, 500)])
def test_products_in_32_bit_and_odd_sizes(device, m, n, k):
    x, w = rnd(m, k), rnd(n, k, seed=1)
    close(ops.linear(x.to(device), w.to(device)), x.double() @ w.double().T, 2e-6)
    xb, wb = x.bfloat16(), w.bfloat16()
    want = xb.double() @ wb.double().T
    close(ops.linear(xb.to(device), wb.to(device), fp32_out=True), want, 1e-5)
    close(ops.linear(xb.to(device), wb.to(device)), want, 1e-2)


# --------------------------------------------------------------------------- recurrence
def recurrence_case(T, H, d, v, seed=0):
    z = rnd(T, H * (2 * d + v), seed=seed)
    bias, lower = 1.5 + rnd(H * d, seed=seed + 1), 0.95 * torch.rand(H * d, generator=torch.Generator().manual_seed(seed))
    lower[0] = 0.9999                                       # one channel that hardly forgets
    return z, bias, lower, 1 + 0.3 * rnd(v, seed=seed + 2)


def recurrence_want(zv, bias, lower, nw, T, H, d, v, eps):
    u = zv[:, :H * d]
    f = O.forget_gate(zv[:, H * d:2 * H * d], bias.double(), lower.double())
    o = O.recurrence((u * torch.sigmoid(u)).view(T, H, d), f.view(T, H, d), zv[:, 2 * H * d:].view(T, H, v))
    return (O.rms(o, eps) * nw.double()).reshape(T, -1)


@on_devices
@in_dtypes
@pytest.mark.parametrize("H,d,v", [(2, 44, 56), (3, 20, 28), (1, 128, 128), (2, 7, 5), (2, 160, 40), (1, 64, 200)])
def test_recurrence_whole_portions_and_single_tokens_agree(device, dtype, H, d, v):
    T, eps = 45, 1e-5
    z, bias, lower, nw = recurrence_case(T, H, d, v)
    zt, zv = projection(z, "bf16" if dtype == torch.bfloat16 else "f32")
    want = recurrence_want(zv, bias, lower, nw, T, H, d, v, eps)
    dev = lambda t: t.to(device)
    args = dev(bias), dev(lower), dev(nw)
    i32 = lambda *x: torch.tensor(x, dtype=torch.int32, device=device)

    def run(state, lo, hi, step=False, slot=1):
        part = dev(zt[lo:hi])
        p = Proj(part, 0, H * d), Proj(part, H * d, H * d), Proj(part, 2 * H * d, H * v)
        kw = dict(heads=H, dim=d, vdim=v, eps=eps, dtype=dtype, rows=i32(slot))
        if not step:
            kw.update(q_start=i32(0), q_lens=i32(hi - lo))
        return ops.hgrn2(*p, *args, state, i32(hi), **kw)

    new_state = lambda: torch.full((3, *hgrn2_state_shape(H, d, v)), 7.0, device=device)   # a slot that was used before
    for cuts in ([T], [1] * 3 + [2] * 4 + [16, 1, 17], [31, 2, 12], [8, 8, 29]):
        state, outs, lo = new_state(), [], 0
        for n in cuts:
            outs.append(run(state, lo, lo + n))
            lo += n
        close(torch.cat(outs), want, TOL[dtype], f"cuts {cuts}")
        assert (state[0] == 7).all() and (state[2] == 7).all()
    state = new_state()
    outs = [run(state, 0, 30)] + [run(state, t, t + 1, step=True) for t in range(30, T)]
    close(torch.cat(outs), want, TOL[dtype], "prompt then single tokens")
    state = new_state()
    close(torch.cat([run(state, t, t + 1, step=True) for t in range(T)]), want, TOL[dtype], "single tokens")


@on_devices
def test_recurrence_batch_of_unequal_sequences_and_inactive_rows(device):
    H, d, v, eps = 2, 24, 36, 1e-5
    lens = [19, 1, 40]
    cases = [recurrence_case(n, H, d, v, seed=10 * i) for i, n in enumerate(lens)]
    bias, lower, nw = cases[0][1:]
    z = torch.cat([c[0] for c in cases])
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)
    state = torch.full((4, *hgrn2_state_shape(H, d, v)), 3.0, device=device)
    sl = lambda t: (Proj(t, 0, H * d), Proj(t, H * d, H * d), Proj(t, 2 * H * d, H * v))
    kw = dict(heads=H, dim=d, vdim=v, eps=eps, dtype=torch.float32)
    w = [t.to(device) for t in (bias, lower, nw)]
    out = ops.hgrn2(*sl(z.to(device)), *w, state, i32(lens), q_start=i32([0, 19, 20]), q_lens=i32(lens),
                    rows=i32([2, 0, 3]), **kw)
    want = [recurrence_want(c[0].double(), bias, lower, nw, n, H, d, v, eps) for c, n in zip(cases, lens)]
    close(out, torch.cat(want), 2e-5)
    # a decode step of rows 0 and 2, rows 1 and 3 inactive: their states stay
    before = state.clone()
    step = rnd(4, z.shape[1], seed=77)
    out = ops.hgrn2(*sl(torch.stack([step, step * 0]).to(device)), *w, state, i32([2, -1, 20, -1]), **kw)
    more = [torch.cat([cases[1][0], step[0:1]]), torch.cat([cases[0][0], step[2:3]])]
    for row, c in zip((0, 2), more):
        close(out[row], recurrence_want(c.double(), bias, lower, nw, len(c), H, d, v, eps)[-1], 2e-5)
    assert torch.equal(state[[1, 3]], before[[1, 3]])


@on_devices
def test_recurrence_keeps_a_write_over_hundreds_of_tokens(device):
    """A channel whose forget gate is nearly one carries the first token's value to the end; the others see noise only."""
    T, H, d, v, eps = 400, 1, 32, 32, 1e-5
    z = 0.05 * rnd(T, H * (2 * d + v))
    bias, lower = torch.full((d,), 0.0), torch.full((d,), 0.0)
    lower[5] = 0.99
    z[0, 2 * d:] = 400.0 * rnd(v, seed=3)
    z[-1, :d] = 0.0
    z[-1, 5] = 6.0
    nw = torch.ones(v)
    want = recurrence_want(z.double(), bias, lower, nw, T, H, d, v, eps)[-1]
    first = z[0, 2 * d:].double()
    assert torch.nn.functional.cosine_similarity(want, first, dim=0) > 0.9
    i32 = lambda *x: torch.tensor(x, dtype=torch.int32, device=device)
    state = torch.zeros((1, *hgrn2_state_shape(H, d, v)), device=device)
    zz = z.to(device)
    out = None
    for lo, hi in ((0, 3), (3, 300), (300, T)):
        part = zz[lo:hi]
        out = ops.hgrn2(Proj(part, 0, d), Proj(part, d, d), Proj(part, 2 * d, v), bias.to(device), lower.to(device),
                        nw.to(device), state, i32(hi), heads=H, dim=d, vdim=v, eps=eps, q_start=i32(0),
                        q_lens=i32(hi - lo), rows=i32(0), dtype=torch.float32)
    close(out[-1], want, 1e-4)


# --------------------------------------------------------------------------- rotation, score maps
@on_devices
@pytest.mark.parametrize("scaling", [None, dict(factor=4.0, original=64, fast=8.0, slow=1.0),
                                     dict(factor=2.0, original=16, fast=1.0, slow=1.0),
                                     dict(factor=8.0, original=4096, fast=32.0, slow=1.0)])
@pytest.mark.parametrize("dim,rdims", [(24, 16), (16, 16), (40, 2)])
def test_rotation_interleaved_partial_and_scaled(device, scaling, dim, rdims):
    T, H, G, vd = 70, 2, 1, 10
    rot = {"base": 1000.0, "dims": rdims, "scaling": scaling}
    rope = C.RopeSpec(1000.0, rdims, **{k: v for k, v in (scaling or {}).items()})
    freq, mult = C.rope_frequencies(rope)
    wf, wm = O.yarn(rot)
    assert torch.allclose(freq, wf) and abs(mult - wm) < 1e-12
    table = ops.rope_table(rdims, 128, inv_freq=freq, scaling=mult, device=device)
    spec = MapsSpec(H, G, dim, vd, 1.0, maps=2, tiled=False)
    z = rnd(T, 2 * dim * (H + G) + vd)
    kc = torch.zeros((4, G, 32, 2 * spec.dim_p), device=device)
    vc = torch.zeros((4, G, 32, spec.vdim_p), device=device)
    order = torch.randperm(4 * 32, generator=torch.Generator().manual_seed(1))[:T].to(torch.int32)
    order[7] = -1                                                   # a token that is not stored
    pos = torch.arange(T, dtype=torch.int32) + 40
    zz = z.to(device)
    q = ops.maps_append(spec, Proj(zz, 0, 2 * dim * H), Proj(zz, 2 * dim * H, 2 * dim * G),
                        Proj(zz, 2 * dim * (H + G), vd), table, pos.to(device), order.to(device), kc, vc)
    want = O.rotate(z[:, :2 * dim * H].double().view(T, H, 2, dim), rot, pos)
    close(q.view(T, H, 2, spec.dim_p)[..., :dim], want, 2e-6)
    wk = O.rotate(z[:, 2 * dim * H:2 * dim * (H + G)].double().view(T, G, 2, dim), rot, pos)
    keep = order >= 0
    got = kc.cpu()[(order // 32).long(), :, (order % 32).long()][keep]
    close(got.view(-1, G, 2, spec.dim_p)[..., :dim], wk[keep], 2e-6)
    close(vc.cpu()[(order // 32).long(), 0, (order % 32).long(), :vd][keep], z[keep, 2 * dim * (H + G):].double(), 1e-6)


class MapsCase:
    """Queries, keys and values of several sequences in a paged cache with scattered blocks."""

    def __init__(self, lens, H, G, d, v, device, dtype, softcap=0.0, std=1.0, seed=0, diff=0.35, lam=0.6):
        self.spec = MapsSpec(H, G, d, v, d ** -0.5, maps=2, softcap=softcap, lam=lam, out_scale=1 - diff, eps=1e-5,
                             tiled=dtype == torch.bfloat16)
        self.diff, self.device, self.dtype, self.lens = diff, device, dtype, lens
        self.q = [rnd(n, H, 2, d, seed=seed + 3 * i, std=std).to(dtype) for i, n in enumerate(lens)]
        self.k = [rnd(n, G, 2, d, seed=seed + 3 * i + 1, std=std).to(dtype) for i, n in enumerate(lens)]
        self.v = [rnd(n, G, v, seed=seed + 3 * i + 2).to(dtype) for i, n in enumerate(lens)]

    def fill(self):
        s = self.spec
        pages = [(n + 31) // 32 for n in self.lens]
        total = sum(pages) + 3
        perm = torch.randperm(total, generator=torch.Generator().manual_seed(9)).tolist()
        # pages hold values of earlier owners (finite); padding columns are zero
        kc, vc = torch.zeros((total, s.kv_heads, 32, 2 * s.dim_p)), torch.zeros((total, s.kv_heads, 32, s.vdim_p))
        kc.view(total, -1, 32, 2, s.dim_p)[..., :s.dim] = 9.0
        vc[..., :s.vdim] = -50.0
        self.table = torch.zeros((len(self.lens), max(pages) + 2), dtype=torch.int32)
        for b, n in enumerate(self.lens):
            for j in range(pages[b]):
                blk = perm.pop()
                self.table[b, j] = blk
                m = min(32, n - 32 * j)
                kc.view(total, -1, 32, 2, s.dim_p)[blk, :, :m, :, :s.dim] = self.k[b][32 * j:32 * j + m].float().transpose(0, 1)
                vc[blk, :, :m, :s.vdim] = self.v[b][32 * j:32 * j + m].float().transpose(0, 1)
        self.kc, self.vc = kc.to(self.device, self.dtype), vc.to(self.device, self.dtype)
        return self

    def want(self, b):
        s, pick = self.spec, torch.arange(self.spec.heads) // (self.spec.heads // self.spec.kv_heads)
        q, k, v = (t[b].double() for t in (self.q, self.k, self.v))
        a = [O.score_map(q[:, :, i], k[:, pick, i], v[:, pick], s.scale, s.softcap) for i in (0, 1)]
        return O.combine(a[0], a[1], s.lam, self.diff, s.eps).reshape(len(q), -1)

    def run(self, parts, step=False):
        """parts: (sequence, first, end) of the new tokens; step: the decode form."""
        s = self.spec
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=self.device)
        q = torch.zeros((sum(e - f for _, f, e in parts), s.heads, 2, s.dim_p))
        o, starts = 0, []
        for b, f, e in parts:
            starts.append(o)
            q[o:o + e - f, :, :, :s.dim] = self.q[b][f:e].float()
            o += e - f
        q = q.reshape(o, s.heads, -1).to(self.device, self.dtype)
        rows = [b for b, _, _ in parts]
        kw = {} if step else dict(q_start=i32(starts), q_lens=i32([e - f for _, f, e in parts]),
                                  max_q_len=max(e - f for _, f, e in parts))
        return ops.maps_attention(s, q, self.kc, self.vc, self.table[rows].to(self.device), i32([e for _, _, e in parts]), **kw)


SIZES = [(6, 3, 28, 64), (4, 4, 24, 40), (6, 1, 64, 128), (2, 1, 48, 80), (20, 2, 16, 128), (3, 3, 64, 64), (2, 2, 96, 72)]


@on_devices
@in_dtypes
@pytest.mark.parametrize("softcap", [0.0, 4.0])
@pytest.mark.parametrize("H,G,d,v", SIZES)
def test_score_maps_in_prompts_and_single_tokens(device, dtype, softcap, H, G, d, v):
    lens = [1, 33, 150, 290]
    c = MapsCase(lens, H, G, d, v, device, dtype, softcap, std=1.3).fill()
    want = [c.want(b) for b in range(len(lens))]
    close(c.run([(b, 0, n) for b, n in enumerate(lens)]), torch.cat(want), TOL[dtype], "whole prompts")
    parts = [(2, 31, 33), (3, 100, 289), (1, 32, 33), (0, 0, 1)]
    close(c.run(parts), torch.cat([want[b][f:e] for b, f, e in parts]), TOL[dtype], "portions")
    for back in (1, 2, 20, 33):
        rows = [(b, n - back, n - back + 1) for b, n in enumerate(lens) if n >= back]
        got = c.run(rows, step=True)
        close(got, torch.stack([want[b][f] for b, f, _ in rows]), TOL[dtype], f"single tokens {back} from the end")


@on_devices
@in_dtypes
def test_score_cap_forms_agree_around_their_limit(device, dtype):
    """Rows with small scores and rows with scores far above the cap (both evaluations of the cap) in one tile."""
    c = MapsCase([140], 2, 1, 32, 64, device, dtype, softcap=3.0, std=1.0)
    c.q[0][::7] = c.q[0][::7] * 12
    c.k[0][5] = c.k[0][5] * 6
    c.q[0][64:96] = c.q[0][64:96] * 0.1
    c.fill()
    want = c.want(0)
    close(c.run([(0, 0, 140)]), want, TOL[dtype])
    close(c.run([(0, 139, 140)], step=True), want[139:], TOL[dtype])


@on_devices
@in_dtypes
@pytest.mark.parametrize("key", [0, 31, 32, 127, 128, 255, 256, 380])
def test_one_far_key_of_hundreds_is_found_by_its_map_only(device, dtype, key):
    """One key fits the last queries of map 1 only; its value is the answer when map 1 dominates the combination."""
    n, d, v = 390, 32, 64
    c = MapsCase([n], 2, 1, d, v, device, dtype, std=0.3, lam=3.0)
    target = rnd(d, seed=42)
    target = (8 * target / target.norm()).to(dtype)
    c.k[0][key, 0, 1] = target
    for qpos in (key, min(key + 1, n - 1), n - 1):
        c.q[0][qpos, :, 1] = target * 1.5
    c.fill()
    want = c.want(0)
    close(c.run([(0, 0, n)]), want, TOL[dtype])
    for qpos in (key, min(key + 1, n - 1), n - 1):
        got = c.run([(0, qpos, qpos + 1)], step=True)
        close(got, want[qpos:qpos + 1], TOL[dtype])
        if qpos >= 3:
            head = want[qpos, :v]
            assert torch.nn.functional.cosine_similarity(head, -c.v[0][key, 0].double(), dim=0) > 0.9
    if key > 0:                     # the position before the key does not see it
        close(c.run([(0, key - 1, key)], step=True), want[key - 1:key], TOL[dtype])


@on_devices
def test_inactive_rows_of_a_decode_step_write_zeros(device):
    c = MapsCase([40, 70], 6, 2, 32, 64, device, torch.bfloat16).fill()
    want = c.want(1)
    s = c.spec
    q = torch.zeros((3, s.heads, 2 * s.dim_p), dtype=torch.bfloat16)
    q[1] = c.q[1][69].reshape(s.heads, -1)
    table = torch.stack([c.table[0], c.table[1], c.table[0]]).to(device)
    out = ops.maps_attention(s, q.to(device), c.kc, c.vc, table, torch.tensor([-1, 70, -1], dtype=torch.int32, device=device))
    close(out[1], want[69], 2e-2)
    assert (out[[0, 2]] == 0).all()
