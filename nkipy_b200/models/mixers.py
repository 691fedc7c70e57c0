"""Token mixers of the layer-by-layer decoders (models/hybrid.py).

A mixer owns the rows it puts into its layer's input projection (`w_in`), its entries of the cache (paged keys and values
or per-sequence states), its output projection (`w_o`), and the step in between: `run` takes the input projection's result
and returns the operand of the output projection, or, where a mixer has no single output projection (`w_o` None), the branches
of the residual.  A new kind of layer is a new class here beside a spec in config.py.
"""

from __future__ import annotations

from typing import List, Union

import torch

from .. import ops
from ..ops import Branch, Decay, HeadRecurrence, LatentSpec, MapsSpec, Proj, ShortConv
from ..ops.linear_attention import linear_state_shape
from ..ops.mixers import hgrn2_state_shape
from .kv_cache import KVLayer, StateLayer


class Tensors:
    """The tensors under one prefix, in the forms the layers keep: fp32 vectors and stacked matrices of the model's type."""

    def __init__(self, get, prefix: str, dtype: torch.dtype):
        self.get, self.prefix, self.dtype = get, prefix, dtype

    def under(self, prefix: str) -> "Tensors":
        return Tensors(self.get, self.prefix + prefix, self.dtype)

    def raw(self, name: str) -> torch.Tensor:
        return self.get(self.prefix + name)

    def f32(self, name: str, offset: float = 0.0) -> torch.Tensor:
        return (self.raw(name).float() + offset).contiguous()

    def mat(self, *names: str) -> torch.Tensor:
        return torch.cat([self.raw(n).to(self.dtype) for n in names]).contiguous()

    def stack(self, *names: str) -> torch.Tensor:
        return torch.stack([self.raw(n).to(self.dtype) for n in names]).contiguous()


def columns(y: Union[torch.Tensor, Proj], widths: List[int]) -> List[Proj]:
    """Slices of a projection's result (or of a slice of it) of the given widths, one after the other."""
    t, c = (y.t, y.col) if isinstance(y, Proj) else (y, 0)
    out = []
    for w in widths:
        out.append(Proj(t, c, w))
        c += w
    return out


def padded_rows(w: torch.Tensor, to: int = 8) -> torch.Tensor:
    """w [N, K] filled up with zero rows to a multiple of `to`."""
    n = -w.shape[0] % to
    return torch.cat([w, w.new_zeros((n, w.shape[1]))]).contiguous() if n else w


class Hgrn2Mixer:
    """Linear recurrence with a forget gate."""

    def __init__(self, spec, t: Tensors, eps: float):
        self.spec, self.eps = spec, eps
        self.w_in, self.w_o = t.mat("q", "f", "v"), t.mat("o")
        self.widths = [spec.heads * spec.dim, spec.heads * spec.dim, spec.heads * spec.vdim]
        self.f_bias, self.lower, self.norm = t.f32("f.b"), t.f32("lower"), t.f32("norm")

    def entries(self):
        return [StateLayer(hgrn2_state_shape(self.spec.heads, self.spec.dim, self.spec.vdim))]

    def run(self, model, y, h, entry, cache, b):
        m = self.spec
        return ops.hgrn2(*columns(y, self.widths), self.f_bias, self.lower, self.norm, cache.state[entry], b.context_lens,
                         heads=m.heads, dim=m.dim, vdim=m.vdim, eps=self.eps, q_start=b.q_start, q_lens=b.q_lens,
                         rows=b.rows, dtype=model.dtype)


class MapsMixer:
    """Differential attention: two score maps per head, interleaved partial rotation."""

    def __init__(self, spec, t: Tensors, eps: float):
        self.spec = spec
        self.w_in, self.w_o = t.mat("q", "k", "v"), t.mat("o")
        self.widths = [spec.heads * 2 * spec.dim, spec.kv_heads * 2 * spec.dim, spec.kv_heads * spec.vdim]
        dot = lambda a, b: float(torch.exp((t.raw(a).double() * t.raw(b).double()).sum()))
        lam = dot("lq1", "lk1") - dot("lq2", "lk2") + spec.diff
        self.maps = MapsSpec(spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.scale, maps=2, softcap=spec.softcap,
                             lam=lam, out_scale=1.0 - spec.diff, eps=eps, tiled=t.dtype == torch.bfloat16)

    def entries(self):
        return [KVLayer(self.spec.kv_heads, self.maps.maps * self.maps.dim_p, self.maps.vdim_p)]

    def run(self, model, y, h, entry, cache, b):
        q = ops.maps_append(self.maps, *columns(y, self.widths), model.rope_table(self.spec.rope), b.positions, b.slots,
                            cache.k[entry], cache.v[entry])
        return ops.maps_attention(self.maps, q, cache.k[entry], cache.v[entry], b.block_table, b.context_lens,
                                  q_start=b.q_start, q_lens=b.q_lens, max_q_len=b.max_q_len)


class LinearAttentionMixer:
    """Gated linear attention."""

    def __init__(self, spec, t: Tensors, eps: float):
        self.spec, self.eps = spec, eps
        self.w_in, self.w_o = t.mat("q", "k", "v", "g", "a1"), t.mat("o")
        c, n = spec.heads * spec.dim, spec.heads * spec.vdim
        self.w_decay, self.decay_bias, self.norm = t.mat("a2"), t.f32("a2.b"), t.f32("norm")
        self.widths = [c, c, n, n, self.w_decay.shape[1]]

    def entries(self):
        return [StateLayer(linear_state_shape(self.spec.heads, self.spec.dim, self.spec.vdim))]

    def run(self, model, y, h, entry, cache, b):
        m = self.spec
        q, k, v, g, a = columns(y, self.widths)
        decay = Decay("sigmoid_root", a, self.w_decay, self.decay_bias, tau=m.tau)
        return ops.linear_attention(q, k, v, decay, g, self.norm, cache.state[entry], b.context_lens, heads=m.heads,
                                    dim=m.dim, vdim=m.vdim, eps=self.eps, q_scale=m.dim ** -0.5, q_start=b.q_start,
                                    q_lens=b.q_lens, rows=b.rows, dtype=model.dtype)


class WindowAttentionMixer:
    """Grouped-query attention over a sliding window, queries and keys normed over all heads, sigmoid-gated heads."""

    def __init__(self, spec, t: Tensors, eps: float, scale: float = 1.0):
        self.spec, self.scale = spec, scale
        self.w_in, self.w_o = t.mat("q", "k", "v", "g"), t.mat("o")
        self.widths = [spec.heads * spec.dim, spec.kv_heads * spec.dim, spec.kv_heads * spec.vdim, spec.heads * spec.vdim]
        self.q_norm, self.k_norm = t.f32("q.norm"), t.f32("k.norm")
        self.maps = MapsSpec(spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.scale, maps=1, eps=eps,
                             window=spec.window, tiled=t.dtype == torch.bfloat16)

    def entries(self):
        return [KVLayer(self.spec.kv_heads, self.maps.dim_p, self.maps.vdim_p)]

    def run(self, model, y, h, entry, cache, b, out=None):
        q, k, v, g = columns(y, self.widths)
        kc, vc = cache.k[entry], cache.v[entry]
        q = ops.row_norm_append(self.maps, q, k, v, self.q_norm, self.k_norm, b.slots, kc, vc)
        o = ops.heads_attention(self.maps, q, kc, vc, b.block_table, b.context_lens, q_start=b.q_start, q_lens=b.q_lens,
                                max_q_len=b.max_q_len)
        return ops.gate_heads(o, g, "sigmoid", scale=self.scale, out=out)


class ChunkAttentionMixer:
    """Grouped-query attention inside chunks of positions, one gate per head.  With `kv_from` its cache entry is that of
    another layer, whose keys and values it reads with its own queries."""

    def __init__(self, spec, t: Tensors, eps: float):
        self.spec = spec
        own = spec.kv_from is None
        names = ("q", "k", "v") if own else ("q",)
        self.w_in, self.w_o = t.mat(*names, "g"), t.mat("o")
        self.widths = [spec.heads * spec.dim, spec.kv_heads * spec.dim, spec.kv_heads * spec.vdim][:len(names)] + [spec.heads]
        self.bias = torch.cat([t.f32(n + ".b") for n in names]).contiguous()
        self.maps = MapsSpec(spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.scale, maps=1, eps=eps, chunk=spec.chunk,
                             tiled=t.dtype == torch.bfloat16)

    def entries(self):
        return [KVLayer(self.spec.kv_heads, self.maps.dim_p, self.maps.vdim_p)] if self.spec.kv_from is None else []

    def run(self, model, y, h, entry, cache, b):
        q, *kv, g = columns(y, self.widths)
        kc, vc = cache.k[entry], cache.v[entry]
        q = ops.rope_norm_append(self.maps, q, *(kv or (None, None)), self.bias, model.rope_table(self.spec.rope), b.positions,
                                 b.slots, kc, vc)
        o = ops.heads_attention(self.maps, q, kc, vc, b.block_table, b.context_lens, q_start=b.q_start, q_lens=b.q_lens,
                                max_q_len=b.max_q_len)
        return ops.gate_heads(o, g, "sigmoid")


class LatentAttentionMixer:
    """Latent attention with a sink and a gate per head.  Small batches attend to the cached latents: the queries are folded
    through the keys' up projection, and the values' up projection is applied to the mixtures of latents.  Large ones expand the
    keys and values of the visible tokens, which takes fewer operations per query."""

    def __init__(self, spec, t: Tensors, eps: float):
        self.spec = spec
        H, R = spec.heads, spec.kv_rank
        self.w_in, self.w_o = t.mat("dq", "dkv", "g"), t.mat("o")
        self.widths = [spec.q_rank, R + spec.rot, H]
        self.w_uq = t.mat("uq")
        self.w_up = t.mat("uk", "uv")                                                    # [H dim + H vdim, R]
        self.w_uk = self.w_up[:H * spec.dim].reshape(H, spec.dim, R).transpose(1, 2).contiguous()
        self.w_uv = self.w_up[H * spec.dim:].reshape(H, spec.vdim, R)
        self.q_norm, self.kv_norm, self.sink = t.f32("dq.norm"), t.f32("dkv.norm"), t.f32("sink")
        self.latent = LatentSpec(H, spec.dim, spec.rot, spec.vdim, R, spec.q_rank, spec.scale, spec.window, eps,
                                 tiled=t.dtype == torch.bfloat16)

    def weights(self):
        return [self.w_uq, self.w_up]

    def entries(self):
        return [KVLayer(1, self.latent.row, 0)]

    def run(self, model, y, h, entry, cache, b):
        s, (q, kv, g) = self.latent, columns(y, self.widths)
        table, rows = model.rope_table(self.spec.rope), cache.k[entry]
        T = h.shape[0]
        c = ops.latent_append(s, q, kv, self.q_norm, self.kv_norm, table, b.positions, b.slots, rows)
        up = Proj(model.project(c, self.w_uq), 0, self.w_uq.shape[0])
        if b.q_lens is not None and not model.is_small(h) and s.slabs is not None:
            q = torch.empty((T, s.heads, 64 * s.slabs[0]), dtype=model.dtype, device=h.device)
            ops.latent_queries(s, up, table, b.positions, q[..., :-64], q[..., -64:])
            pages, base = b.visible_pages(s.window)
            c, r = ops.latent_gather(s, rows, pages, (s.rot + 7) // 8 * 8)
            kv = model.project(c, self.w_up)
            o = ops.latent_prefill(s, q, kv, r, base, b.q_start, b.q_lens, b.context_lens, b.max_q_len, self.sink)
            return ops.gate_heads(o, g, "sigmoid")
        plain = torch.empty((s.heads, T, s.dim), dtype=model.dtype, device=h.device)
        q = torch.empty((s.heads, T, s.row), dtype=model.dtype, device=h.device)
        ops.latent_queries(s, up, table, b.positions, plain.transpose(0, 1), q.transpose(0, 1)[..., s.rank:])
        ops.head_linear(plain, self.w_uk, out=q[..., :s.rank])
        o = ops.latent_attention(s, q, rows, b.block_table, b.context_lens, q_start=b.q_start, q_lens=b.q_lens,
                                 sinks=self.sink)
        return ops.gate_heads(ops.head_linear(o, self.w_uv).transpose(0, 1), g, "sigmoid")


class TimeMixMixer:
    """RWKV-style time mixing.  Its projections read mixes of neighbouring tokens and not h, so it has no rows in the
    layer's input projection."""

    def __init__(self, spec, t: Tensors, eps: float, scale: float = 1.0):
        self.spec, self.eps, self.scale = spec, eps, scale
        self.w_in, self.widths, self.w_o = None, [], t.mat("o")
        self.w_each, self.w_narrow, self.w_decay = t.stack("r", "k", "v", "g"), t.mat("w1"), t.mat("w2")
        self.mu = torch.stack([t.f32("mu." + n) for n in "rkvgw"]).contiguous()
        self.decay_bias, self.bonus, self.norm = t.f32("w0"), t.f32("u").reshape(-1).contiguous(), t.f32("norm")

    def entries(self):
        return [StateLayer(linear_state_shape(self.spec.heads, self.spec.dim, self.spec.dim)), StateLayer((self.mu.shape[1],))]

    def run(self, model, y, h, entry, cache, b, out=None):
        m = self.spec
        x = ops.token_mix(h, self.mu, cache.state[entry + 1], b.context_lens, q_start=b.q_start, q_lens=b.q_lens,
                          rows=b.rows)
        r, k, v, g = model.project_each(x[:4], self.w_each)
        narrow = model.project(x[4], self.w_narrow)
        decay = Decay("double_exp", Proj(narrow, 0, self.w_narrow.shape[0]), self.w_decay, self.decay_bias, act="tanh")
        return ops.linear_attention(r, k, v, decay, g, self.norm, cache.state[entry], b.context_lens, heads=m.heads,
                                    dim=m.dim, vdim=m.dim, eps=self.eps, bonus=self.bonus, scale=self.scale,
                                    q_start=b.q_start, q_lens=b.q_lens, rows=b.rows, dtype=model.dtype, out=out)


class ParallelMixer:
    """Two mixers on the same input.  Their constant weights are applied to the operands of the output projections, which
    then are one product over the joined operands."""

    def __init__(self, spec, t: Tensors, eps: float):
        self.left = WindowAttentionMixer(spec.left, t.under("left."), eps, spec.left_scale)
        self.right = TimeMixMixer(spec.right, t.under("right."), eps, spec.right_scale)
        self.w_in, self.widths = self.left.w_in, self.left.widths
        self.split = self.left.w_o.shape[1]
        self.w_o = torch.cat([self.left.w_o, self.right.w_o], 1).contiguous()
        self.left.w_o = self.right.w_o = None

    def entries(self):
        return self.left.entries() + self.right.entries()

    def run(self, model, y, h, entry, cache, b):
        out = torch.empty((h.shape[0], self.w_o.shape[1]), dtype=model.dtype, device=h.device)
        self.left.run(model, y, h, entry, cache, b, out=out[:, :self.split])
        self.right.run(model, None, h, entry + 1, cache, b, out=out[:, self.split:])
        return out


class GroupedAttentionMixer:
    """Grouped-query attention with the options of `GroupedAttentionSpec`."""

    def __init__(self, spec, t: Tensors, eps: float):
        self.spec = s = spec
        names = ("q", "k", "v") if s.kv_from is None else ("q",)
        self.w_in, self.w_o = t.mat(*names, *(("g",) if s.gate else ())), t.mat("o")
        self.widths = [s.heads * s.dim, s.kv_heads * s.dim, s.kv_heads * s.vdim][:len(names)] + ([s.heads] if s.gate else [])
        self.bias = torch.cat([t.f32(n + ".b") for n in names]).contiguous() if s.bias else None
        self.o_bias = t.f32("o.b") if s.bias else None
        self.sink = t.f32("sink") if s.sink else None
        dist = (t.f32("r1"), t.f32("r2")) if s.distance else (None, None)
        self.maps = MapsSpec(s.heads, s.kv_heads, s.dim, s.vdim, s.scale, maps=1, softcap=s.softcap, eps=eps, window=s.window,
                             keep_first=s.keep_first if s.window > 0 else 0, dist_a=dist[0], dist_b=dist[1],
                             tiled=t.dtype == torch.bfloat16)

    def entries(self):
        return [KVLayer(self.spec.kv_heads, self.maps.dim_p, self.maps.vdim_p)] if self.spec.kv_from is None else []

    def run(self, model, y, h, entry, cache, b):
        q, *kv = columns(y, self.widths)
        g = kv.pop() if self.spec.gate else None
        kc, vc, rope = cache.k[entry], cache.v[entry], self.spec.rope
        q = ops.rope_norm_append(self.maps, q, *(kv or (None, None)), self.bias, model.rope_table(rope) if rope else None,
                                 b.positions, b.slots, kc, vc, norm=False, interleaved=True)
        o = ops.heads_attention(self.maps, q, kc, vc, b.block_table, b.context_lens, q_start=b.q_start, q_lens=b.q_lens,
                                max_q_len=b.max_q_len, sinks=self.sink)
        return o.flatten(1) if g is None else ops.gate_heads(o, g, "sigmoid")


class DeltaMixer:
    """Gated delta rule."""

    def __init__(self, spec, t: Tensors, eps: float):
        c, n, H = spec.kv_heads * spec.dim, spec.heads * spec.vdim, spec.heads
        self.w_in, self.w_o = t.mat("q", "k", "v", "g", "b", "a"), t.mat("o")
        self.widths = [2 * c + n, n, H, H]
        self.conv = ShortConv(torch.cat([t.f32(x + ".conv") for x in "qkv"]).t().contiguous())
        self.norm = t.f32("norm")
        self.rule = HeadRecurrence(H, spec.kv_heads, spec.dim, spec.vdim, 0, c, 2 * c, torch.exp(t.f32("A_log")), t.f32("dt_bias"),
                                   delta=True, q_scale=spec.dim ** -0.5, eps=eps)

    def entries(self):
        return [StateLayer(self.rule.state_shape), StateLayer(self.conv.state_shape)]

    def run(self, model, y, h, entry, cache, b):
        x, gate, strength, decay = columns(y, self.widths)
        return ops.head_recurrence(self.rule, x, self.conv, decay, strength, gate, self.norm, cache.state[entry],
                                   cache.state[entry + 1], b.context_lens, q_start=b.q_start, q_lens=b.q_lens, rows=b.rows,
                                   dtype=model.dtype)


class StateSpaceMixer:
    """Mamba-2."""

    def __init__(self, spec, t: Tensors, eps: float):
        n, c = spec.heads * spec.vdim, spec.groups * spec.state
        self.w_in, self.w_o = t.mat("in"), t.mat("o")
        self.widths, self.parts = [n, n + 2 * c, spec.heads], spec.norm_groups
        self.conv = ShortConv(t.f32("conv").t().contiguous(), t.f32("conv.b"))
        self.norm = t.f32("norm")
        self.rule = HeadRecurrence(spec.heads, spec.groups, spec.state, spec.vdim, n + c, n, 0, torch.exp(t.f32("A_log")),
                                   t.f32("dt_bias"), delta=False, skip=t.f32("D"), eps=eps)

    def entries(self):
        return [StateLayer(self.rule.state_shape), StateLayer(self.conv.state_shape)]

    def run(self, model, y, h, entry, cache, b):
        gate, x, dt = columns(y, self.widths)
        return ops.head_recurrence(self.rule, x, self.conv, dt, None, gate, self.norm, cache.state[entry], cache.state[entry + 1],
                                   b.context_lens, parts=self.parts, q_start=b.q_start, q_lens=b.q_lens, rows=b.rows,
                                   dtype=model.dtype)


class BlendMixer:
    """Two mixers on the same input, each with its own output projection; the mean of their results, RMS-normed over the width.
    Their rows of the input projection are one matrix, each part filled up to whole 16 bytes with zero rows."""

    def __init__(self, spec, t: Tensors, eps: float):
        self.left = GroupedAttentionMixer(spec.left, t.under("left."), eps)
        self.right = StateSpaceMixer(spec.right, t.under("right."), eps)
        self.norms = [t.f32("left.out"), t.f32("right.out")]
        left = padded_rows(self.left.w_in)
        self.w_in, self.w_o = torch.cat([left, self.right.w_in]).contiguous(), None
        self.widths = [left.shape[0], self.right.w_in.shape[0]]
        self.left.w_in = self.right.w_in = None

    def weights(self):
        return [self.left.w_o, self.right.w_o]

    def entries(self):
        return self.left.entries() + self.right.entries()

    def run(self, model, y, h, entry, cache, b):
        left, right = columns(y, self.widths)
        outs = [(self.left, self.left.run(model, left, h, entry, cache, b)),
                (self.right, self.right.run(model, right, h, entry + len(self.left.entries()), cache, b))]
        return [Branch(Proj(model.project(o, m.w_o), 0, m.w_o.shape[0]), scale=0.5, norm=n, shift=getattr(m, "o_bias", None))
                for (m, o), n in zip(outs, self.norms)]


MIXERS = {"hgrn2": Hgrn2Mixer, "attention": MapsMixer, "gla": LinearAttentionMixer, "window": WindowAttentionMixer,
          "rwkv": TimeMixMixer, "parallel": ParallelMixer, "chunk": ChunkAttentionMixer, "latent": LatentAttentionMixer,
          "grouped": GroupedAttentionMixer, "delta": DeltaMixer, "ssd": StateSpaceMixer, "blend": BlendMixer}
