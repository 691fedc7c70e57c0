"""Decoders whose layers are listed one by one: each layer has its own token mixer (models/mixers.py) and feed-forward,
around an fp32 residual stream.  Four kinds of layer:

    gated (Tolenex)       h1 = norm1(x), h2 = norm2(x)
                          x <- x + sigmoid(W_g1 h1 + b1) * mixer(h1) + sigmoid(W_g2 h2 + b2) * feed_forward(h2)
    pre-norm (Mumilorn)   x <- x + mixer(norm1(x)),   then   x <- x + feed_forward(norm2(x))
    sandwich (Redodra)    x <- x + norm1b(mixer(norm1(x))),   then   x <- x + norm2b(feed_forward(norm2(x)))
    parallel (Ligizen)    h = norm1(x);  x <- x + mixer(h) + feed_forward(h),  then  x <- x + norm(token input of x)

A layer is a list of stages; a stage reads norms of the residual and returns the branches that are added to it.  One
kernel per stage (`ops.gated_residual`) sums the branches, applies what precedes a repeated pass of a looped block and
norms the result for the next stage.  With `depth_average` what leaves a layer is a weighted sum of the embedding output and all
layers' results so far, which that kernel computes as well.  The model plugs into the same engine, paged cache and decode graph as
`TransformerLM`.

Batches of at most 128 tokens (decode steps, small mixed steps) run their projections as split-K GEMMs whose fp32
partial sums the next kernel adds up; larger ones as tiled GEMMs with bf16 results and the activation in
the epilogue.  Attention and recurrence have their own kernels for "one new token per sequence" and for packed
prompts; both read and leave the same cache and state.

`dtype` float32 runs the whole model in true 32-bit (weights, activations, cache; products on the CUDA cores).
"""

from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import ops
from ..ops import Branch, Norm, Proj
from ..ops.mixers import History
from ..parallel.comm import TPGroup
from .config import LayerSpec, ModelConfig, RopeSpec, rope_frequencies
from .kv_cache import BLOCK_SIZE, PagedKVCache
from .mixers import MIXERS, Tensors, padded_rows
from .moe import RoutedExperts
from .transformer import pick_splits

SMALL_BATCH = 128


class Stage:
    """norms: the residual's norms it reads (weights of RMS norms, or `ops.Norm`); run(h, entry, cache, batch) -> branches;
    post: what their sum passes before it is added."""
    __slots__ = ("norms", "run", "post")

    def __init__(self, norms, run, post: Optional[Norm] = None):
        self.norms, self.run, self.post = norms, run, post


class GatedLayer:
    """Mixer and gated feed-forward beside each other.  Input projections stacked: w_in1 = [mixer inputs; gate 1],
    w_in2 = [gate; up; gate 2]."""

    def __init__(self, model: "HybridLM", spec: LayerSpec, t: Tensors):
        cfg = model.cfg
        self.model, self.spec, self.width = model, spec, cfg.hidden_size
        self.mixer = MIXERS[spec.mixer.kind](spec.mixer, t.under("mix."), cfg.rms_eps)
        self.w_in1 = torch.cat([self.mixer.w_in, t.mat("rg1")]).contiguous()
        self.mixer.w_in = None
        self.gate_bias = [t.f32("rg1.b")]
        norms = [t.f32("norm1", cfg.norm_offset)]
        if spec.ff:
            norms.append(t.f32("norm2", cfg.norm_offset))
            self.w_in2 = t.mat("mlp.gate", "mlp.up", "rg2")
            self.w_down = t.mat("mlp.down")
            self.gate_bias.append(t.f32("rg2.b"))
        if sum(self.mixer.widths) + cfg.hidden_size != self.w_in1.shape[0]:
            raise ValueError("projection sizes do not fit the configuration")
        self.stages = [Stage(norms, self._run)]

    def weights(self):
        return [self.w_in1, self.mixer.w_o] + ([self.w_in2, self.w_down] if self.spec.ff else [])

    def _feed_forward(self, h: torch.Tensor):
        """(down projection, gate slice) of the feed-forward branch."""
        ff, width, m = self.spec.ff, self.width, self.model
        if x_small(h):
            y = m.project(h, self.w_in2)
            act = ops.gated_act(Proj(y, 0, ff), Proj(y, ff, ff), self.spec.act, dtype=h.dtype)
            gate = Proj(y, 2 * ff, width)
        else:
            act = ops.linear(h, self.w_in2[:2 * ff], gated=True, act=self.spec.act, swap=False)
            gate = Proj(ops.linear(h, self.w_in2[2 * ff:], swap=False), 0, width)
        return Proj(m.project(act, self.w_down), 0, width), gate

    def _run(self, h, entry, cache, b) -> List[Branch]:
        m, width = self.model, self.width
        y = m.project(h[0], self.w_in1)
        mixed = self.mixer.run(m, y, h[0], entry, cache, b)
        branches = [Branch(Proj(m.project(mixed, self.mixer.w_o), 0, width), Proj(y, sum(self.mixer.widths), width),
                           self.gate_bias[0])]
        if self.spec.ff:
            branches.append(Branch(*self._feed_forward(h[1]), self.gate_bias[1]))
        return branches


class DenseMLP:
    """down(act(up h)); xIELU's two parameters are the tensor `act`, through softplus."""

    def __init__(self, act: str, t: Tensors):
        self.act, self.up, self.down = act, t.mat("up"), t.mat("down")
        if act == "xielu":
            p, q = torch.nn.functional.softplus(t.raw("act").double(), threshold=100.0).tolist()
            self.act = ops.Act("xielu", p, 0.5 + q)

    def weights(self):
        return [self.up, self.down]

    def run(self, model: "HybridLM", h: torch.Tensor) -> List[Branch]:
        if x_small(h):
            a = ops.activation(Proj(model.project(h, self.up), 0, self.up.shape[0]), self.act, dtype=h.dtype)
        else:
            a = ops.linear(h, self.up, swap=False, out_act=self.act)
        return [Branch(Proj(model.project(a, self.down), 0, h.shape[1]))]


class GatedMLP:
    """down(act(gate h) * up h).  `w_wide` holds [gate; up] as rows for the input projection of a layer whose sublayers share
    their input."""

    def __init__(self, act: str, t: Tensors):
        self.act, self.w_wide, self.w_narrow, self.down = act, t.mat("gate", "up"), None, t.mat("down")

    def weights(self):
        return [self.w_wide, self.down]

    def run(self, model: "HybridLM", h: torch.Tensor, wide: Optional[Proj] = None, narrow=None) -> List[Branch]:
        if wide is None and x_small(h):
            wide = Proj(model.project(h, self.w_wide), 0, self.w_wide.shape[0])
        if wide is not None:
            n = wide.width // 2
            a = ops.gated_act(Proj(wide.t, wide.col, n), Proj(wide.t, wide.col + n, n), self.act, dtype=h.dtype)
        else:
            a = ops.linear(h, self.w_wide, gated=True, act=self.act, swap=False)
        return [Branch(Proj(model.project(a, self.down), 0, h.shape[1]))]


class PreNormLayer:
    """Mixer, then feed-forward (dense or routed), each on its own norm of the residual."""

    def __init__(self, model: "HybridLM", spec: LayerSpec, t: Tensors):
        cfg = model.cfg
        self.model, self.width = model, cfg.hidden_size
        self.mixer = MIXERS[spec.mixer.kind](spec.mixer, t.under("mix."), cfg.rms_eps)
        self.mlp = None
        if spec.experts is not None:
            self.mlp = RoutedExperts(spec.experts, t.under("mlp."))
        elif spec.ff:
            self.mlp = DenseMLP(spec.act, t.under("mlp."))
        if self.mixer.w_in is not None and sum(self.mixer.widths) != self.mixer.w_in.shape[0]:
            raise ValueError("projection sizes do not fit the configuration")
        self.stages = [Stage([t.f32("norm1", cfg.norm_offset)], self._mix)]
        if self.mlp is not None:
            self.stages.append(Stage([t.f32("norm2", cfg.norm_offset)], lambda h, *_: self.mlp.run(model, h[0])))

    def weights(self):
        ws = [self.mixer.w_in, self.mixer.w_o, getattr(getattr(self.mixer, "right", None), "w_each", None)]
        return [w for w in ws if w is not None] + (self.mlp.weights() if self.mlp is not None else [])

    def _mix(self, h, entry, cache, b) -> List[Branch]:
        m = self.model
        y = m.project(h[0], self.mixer.w_in) if self.mixer.w_in is not None else None
        return [Branch(Proj(m.project(self.mixer.run(m, y, h[0], entry, cache, b), self.mixer.w_o), 0, self.width))]


class SandwichLayer:
    """Mixer, then feed-forward, each with a norm of the residual ahead of it and a norm of its result behind it."""

    def __init__(self, model: "HybridLM", spec: LayerSpec, t: Tensors):
        cfg = model.cfg
        self.model, self.width = model, cfg.hidden_size
        self.mixer = mixer = MIXERS[spec.mixer.kind](spec.mixer, t.under("mix."), cfg.rms_eps)
        if sum(mixer.widths) != mixer.w_in.shape[0]:
            raise ValueError("projection sizes do not fit the configuration")
        mixer.w_in = padded_rows(mixer.w_in)
        self.mlp = DenseMLP(spec.act, t.under("mlp.")) if spec.ff else None
        self.stages = [Stage([model.norm(t, "norm1")], self._mix, model.norm(t, "norm1b"))]
        if self.mlp is not None:
            self.stages.append(Stage([model.norm(t, "norm2")], lambda h, *_: self.mlp.run(model, h[0]), model.norm(t, "norm2b")))

    def weights(self):
        ws = [self.mixer.w_in, self.mixer.w_o, *getattr(self.mixer, "weights", list)()]
        return [w for w in ws if w is not None] + (self.mlp.weights() if self.mlp is not None else [])

    def _mix(self, h, entry, cache, b) -> List[Branch]:
        m = self.model
        o = self.mixer.run(m, m.project(h[0], self.mixer.w_in), h[0], entry, cache, b)
        return o if isinstance(o, list) else [Branch(Proj(m.project(o, self.mixer.w_o), 0, self.width))]


class ParallelLayer:
    """Mixer and feed-forward on one norm of the residual, then the layer's token input: a low-rank product of the residual and
    a row of a table that belongs to the token and the layer.

    Small batches run one input projection [feed-forward's wide rows; mixer; feed-forward's narrow rows], each part filled up
    to whole 16 bytes with zero rows; `spans` holds the rows of the parts."""

    def __init__(self, model: "HybridLM", spec: LayerSpec, t: Tensors):
        cfg = model.cfg
        self.model, self.width = model, cfg.hidden_size
        self.mixer = mixer = MIXERS[spec.mixer.kind](spec.mixer, t.under("mix."), cfg.rms_eps)
        self.mlp = None
        if spec.experts is not None:
            self.mlp = RoutedExperts(spec.experts, t.under("mlp."))
        elif spec.ff:
            self.mlp = GatedMLP(spec.act, t.under("mlp."))
        if sum(mixer.widths) != mixer.w_in.shape[0]:
            raise ValueError("projection sizes do not fit the configuration")
        parts = [getattr(self.mlp, "w_wide", None), mixer.w_in, getattr(self.mlp, "w_narrow", None)]
        self.spans, rows, n = [], [], 0
        for w in parts:
            if w is None:
                self.spans.append(None)
                continue
            self.spans.append((n, w.shape[0]))
            pad = -w.shape[0] % 8
            rows += [w] + ([w.new_zeros((pad, w.shape[1]))] if pad else [])
            n += w.shape[0] + pad
        self.w_in = torch.cat(rows).contiguous()
        views = [None if s is None else self.w_in[s[0]:s[0] + s[1]] for s in self.spans]
        start, rows = self.spans[1]
        mixer.w_in = self.w_in[start:start + (rows + 7) // 8 * 8]
        if self.mlp is not None:
            self.mlp.w_wide, self.mlp.w_narrow = views[0], views[2]
        self.stages = [Stage([model.norm(t, "norm1")], self._run)]
        if cfg.token_side:
            self.side_gate, self.side_proj, self.side_norm = t.mat("side.gate"), t.mat("side.proj"), t.f32("side.norm")
            self.stages.append(Stage([Norm()], self._token_input))

    def weights(self):
        ws = [self.w_in, self.mixer.w_o, *getattr(self.mixer, "weights", list)()]
        if self.mlp is not None:
            ws += [w for w in self.mlp.weights() if w is not self.mlp.w_wide and w is not self.mlp.w_narrow]
        return ws + ([self.side_gate, self.side_proj] if self.model.cfg.token_side else [])

    def _run(self, h, entry, cache, b) -> List[Branch]:
        m, h = self.model, h[0]
        wide = narrow = None
        if x_small(h):
            y = m.project(h, self.w_in)
            wide, mix, narrow = [None if s is None else Proj(y, *s) for s in self.spans]
        else:
            mix = Proj(m.project(h, self.mixer.w_in), 0, self.spans[1][1])
        o = self.mixer.run(m, mix, h, entry, cache, b)
        branches = [Branch(Proj(m.project(o, self.mixer.w_o), 0, self.width))]
        return branches if self.mlp is None else branches + self.mlp.run(m, h, wide, narrow)

    def _token_input(self, h, entry, cache, b) -> List[Branch]:
        m, n = self.model, self.side_gate.shape[0]
        z = Proj(m.project(h[0], self.side_gate), 0, n)
        a = ops.gated_act(z, Proj(m.side_table, m.layers.index(self) * n, n), "gelu_tanh", dtype=m.dtype, up_rows=b.ids)
        return [Branch(Proj(m.project(a, self.side_proj), 0, self.width), norm=self.side_norm)]


LAYERS = {"gated": GatedLayer, "pre-norm": PreNormLayer, "sandwich": SandwichLayer, "parallel": ParallelLayer}


class HybridLM:
    """Weights + forward passes; the interface of `TransformerLM` (one rank)."""

    def __init__(self, cfg: ModelConfig, weights: Dict[str, torch.Tensor], tp: Optional[TPGroup] = None, device=None,
                 dtype: torch.dtype = torch.bfloat16):
        self.cfg = cfg
        self.tp = tp or TPGroup.single()
        if self.tp.world_size > 1:
            raise NotImplementedError(f"{cfg.name} runs on one GPU")
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"unsupported dtype {dtype}")
        self.dtype = dtype
        self.device = torch.device(device if device is not None else weights["embed"].device)
        get = lambda name: weights[name].to(self.device)
        self.embed = get("embed").to(dtype).contiguous()
        self.head = self.embed if cfg.tie_embeddings else get("head").to(dtype).contiguous()
        self.final_norm = self.norm(Tensors(get, "final.", dtype), "norm")
        self.side_table = get("side.embed").to(dtype).contiguous() if cfg.token_side else None
        self.layers = [LAYERS[s.block](self, s, Tensors(get, f"l{i}.", dtype)) for i, s in enumerate(cfg.layers)]
        self.runs = cfg.layer_runs()
        self.entry = []                      # first cache entry of every run, or that of the layer whose keys it reads
        n, first = 0, {}
        for i, _ in self.runs:
            source = getattr(cfg.layers[i].mixer, "kv_from", None)
            first[i] = n if source is None else first[source]
            self.entry.append(first[i])
            n += len(self.layers[i].mixer.entries())
        if cfg.depth_average and cfg.loop:
            raise ValueError("a depth average is over layers that run once")
        self.averages = [get(f"l{i}.dwa").float().contiguous() for i in range(len(cfg.layers))] if cfg.depth_average else None
        self.loop_step = get("loop.step").float().contiguous() if cfg.loop else None
        self._rope: Dict[RopeSpec, torch.Tensor] = {}
        self._offsets: Dict[tuple, torch.Tensor] = {}

    def norm(self, t: Tensors, name: str) -> Norm:
        """The model's kind of norm, from the tensors of that name."""
        if self.cfg.tanh_norm:
            return Norm(t.f32(name), t.f32(name + ".b"), alpha=float(t.raw(name + ".alpha")))
        if self.cfg.layer_norm:
            return Norm(t.f32(name), t.f32(name + ".b"), center=True)
        return Norm(t.f32(name, self.cfg.norm_offset))

    # ------------------------------------------------------------------ cache
    def new_cache(self, num_blocks: int, max_batch: int, max_seq_len: int,
                  enable_prefix_sharing: bool = True) -> PagedKVCache:
        max_blocks = (max_seq_len + self.cfg.block_size - 1) // self.cfg.block_size
        self._extend_rope(max_blocks * self.cfg.block_size)
        entries = [e for i, _ in self.runs for e in self.layers[i].mixer.entries()]
        return PagedKVCache.for_layers(entries, num_blocks, max_batch, max_blocks, self.device, self.dtype,
                                       enable_prefix_sharing)

    def _extend_rope(self, positions: int) -> None:
        """cos / sin tables [positions, dims] of every rotation the layers use."""
        specs = [m for layer in self.cfg.layers for m in (layer.mixer, getattr(layer.mixer, "left", None))]
        for rope in (getattr(m, "rope", None) for m in specs):
            if rope is not None and (rope not in self._rope or self._rope[rope].shape[0] < positions):
                freq, mult = rope_frequencies(rope)
                self._rope[rope] = ops.rope_table(rope.dims, positions, inv_freq=freq, scaling=mult, device=self.device)

    def rope_table(self, rope: RopeSpec) -> torch.Tensor:
        return self._rope[rope]

    def weight_bytes(self) -> int:
        ts = [self.embed, self.head] + ([] if self.side_table is None else [self.side_table]) + [t for l in self.layers for t in l.weights()]
        return sum(t.numel() * t.element_size() for t in ts)

    # ------------------------------------------------------------------ layers
    @staticmethod
    def is_small(h: torch.Tensor) -> bool:
        """Whether projections of h come as fp32 (split-K) sums, see `project`."""
        return x_small(h)

    def project(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """fp32 (split-K partials) for small batches, bf16 for large ones, fp32 for 32-bit models."""
        if x.dtype == torch.float32:
            return ops.linear(x, w)
        if x.shape[0] <= SMALL_BATCH:
            splits = pick_splits(w.shape[0], w.shape[1])
            return ops.linear(x, w, splits=splits) if splits > 1 else ops.linear(x, w, fp32_out=True)
        return ops.linear(x, w, swap=False)

    def project_each(self, x: torch.Tensor, w: torch.Tensor) -> List[Proj]:
        """x[i] @ w[i].T for x [M, T, K], w [M, N, K]: one grouped product for small bf16 batches."""
        M, T, K = x.shape
        N = w.shape[1]
        if x_small(x[0]) and x.dtype == torch.bfloat16 and K % 8 == 0:
            if (M, T) not in self._offsets:
                self._offsets[M, T] = torch.arange(0, M * T + 1, T, dtype=torch.int32, device=x.device)
            y = ops.grouped_linear(x.reshape(M * T, K), w, self._offsets[M, T], max_rows_per_group=T)
            return [Proj(y[i * T:(i + 1) * T], 0, N) for i in range(M)]
        return [Proj(self.project(x[i], w[i]), 0, N) for i in range(M)]

    def _forward(self, ids: torch.Tensor, cache: PagedKVCache, b: "Batch", return_hidden: bool = False):
        cfg = self.cfg
        norm = dict(groups=cfg.norm_groups, eps=cfg.rms_eps, dtype=self.dtype)
        start = cfg.loop.start if cfg.loop else -1
        plan = [(r, s) for r, (i, _) in enumerate(self.runs) for s in range(len(self.layers[i].stages))]

        def ahead(n):
            """What is added to the residual before stage n of the plan, and the norms that read it."""
            if n == len(plan):
                return dict(norms=[self.final_norm])
            r, s = plan[n]
            i, t = self.runs[r]
            pre = dict(norms=self.layers[i].stages[s].norms)
            if s == 0 and t >= 0 and i == start:
                pre["add_row"] = self.loop_step[t]
                if t > 0:
                    pre["add_mat"] = embedded
            return pre

        first = ahead(0)
        rows = None                          # results that later layers average: the embedding output, then every layer's
        if cfg.depth_average:
            rows = torch.empty((len(self.runs), ids.numel(), cfg.hidden_size), dtype=torch.float32, device=self.embed.device)
        x, h = ops.gated_residual(None, ids=ids, table=self.embed, scale=cfg.embedding_scale,
                                  norms=[] if "add_row" in first else first["norms"], out=None if rows is None else rows[0], **norm)
        embedded = x
        if "add_row" in first:
            x, h = ops.gated_residual(x, **first, **norm)
        taps = []
        for n, (r, s) in enumerate(plan):
            stages = self.layers[self.runs[r][0]].stages
            branches = stages[s].run(h, self.entry[r], cache, b)
            how = dict(post=stages[s].post)
            if s == len(stages) - 1:
                if rows is not None:
                    how["history"] = History(rows, r + 1, self.averages[r], store=r + 1 < len(rows))
                if return_hidden:
                    taps.append(ops.gated_residual(x, branches, eps=cfg.rms_eps, **how)[0])
            x, h = ops.gated_residual(x, branches, **ahead(n + 1), **how, **norm)
        return (h[0], taps) if return_hidden else h[0]

    # ------------------------------------------------------------------ the engine's entry points
    def prefill(self, ids, positions, slots, cache, block_table, q_start, q_lens, context_lens, max_q_len,
                return_hidden: bool = False, rows: Optional[torch.Tensor] = None, spans=None):
        """Packed step over the new tokens of several sequences (whole prompts, portions of prompts, single tokens);
        rows[b] is the batch row (state slot) of sequence b, spans its [first new position, context length) on the host (read
        back from the device when not given and needed).  Returns the final-normed hidden states [T, W] (and the
        residual stream after every layer run)."""
        return self._forward(ids, cache, Batch(positions, slots, block_table, context_lens, q_start, q_lens, max_q_len,
                                               rows, ids, spans), return_hidden)

    def decode_step(self, ids, positions, slots, cache, block_table, context_lens, return_hidden: bool = False):
        """One new token for every batch row; rows with a negative context length are inactive."""
        return self._forward(ids, cache, Batch(positions, slots, block_table, context_lens, ids=ids), return_hidden)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits [rows, vocab]."""
        z = ops.linear(hidden, self.head, fp32_out=True)
        return ops.softcap(z, self.cfg.logit_softcap) if self.cfg.logit_softcap > 0 else z

    def greedy(self, hidden: torch.Tensor, out_ids: Optional[torch.Tensor] = None) -> torch.Tensor:
        return ops.argmax(self.logits(hidden), out_ids=out_ids)

    def close(self) -> None:
        pass


class Batch:
    """The tokens of a step, where they sit (cache slots, block tables) and how they are grouped into sequences (q_lens
    None: one per batch row)."""
    __slots__ = ("positions", "slots", "block_table", "context_lens", "q_start", "q_lens", "max_q_len", "rows", "ids",
                 "_spans", "_pages")

    def __init__(self, positions, slots, block_table, context_lens, q_start=None, q_lens=None, max_q_len=1, rows=None,
                 ids=None, spans=None):
        self.positions, self.slots, self.block_table, self.context_lens = positions, slots, block_table, context_lens
        self.q_start, self.q_lens, self.max_q_len, self.rows = q_start, q_lens, max_q_len, rows
        self.ids, self._spans, self._pages = ids, spans, {}

    def visible_pages(self, window: int):
        """Cache pages that the new tokens see through a sliding window (0: all before them), sequence by sequence (int32 block
        numbers), and per sequence the row its position 0 has when those pages' tokens follow one another."""
        if window not in self._pages:
            if self._spans is None:
                self._spans = [(c - n, c) for c, n in zip(self.context_lens.tolist(), self.q_lens.tolist())]
            seq, page, base, n = [], [], [], 0
            for b, (first, end) in enumerate(self._spans):
                lo = max(0, first - window + 1) // BLOCK_SIZE if window > 0 else 0
                hi = (end + BLOCK_SIZE - 1) // BLOCK_SIZE
                seq += [b] * (hi - lo)
                page += range(lo, hi)
                base.append((n - lo) * BLOCK_SIZE)
                n += hi - lo
            dev = self.block_table.device
            at = torch.tensor([seq, page], dtype=torch.long).to(dev, non_blocking=True)
            self._pages[window] = (self.block_table[at[0], at[1]].to(torch.int32).contiguous(),
                                   torch.tensor(base, dtype=torch.int32).to(dev, non_blocking=True))
        return self._pages[window]


def x_small(h: torch.Tensor) -> bool:
    """Whether projections of h come as fp32 sums and leave what follows them to a kernel of its own."""
    return h.dtype == torch.float32 or h.shape[0] <= SMALL_BATCH
