"""Decoder whose layers are listed one by one: attention with score maps or a linear recurrence, each beside a dense
feed-forward, around an fp32 residual stream (the Tolenex design).

A layer reads the residual once and updates it once:

    h1 = norm1(x), h2 = norm2(x)
    x <- x + sigmoid(W_g1 h1 + b1) * mixer(h1) + sigmoid(W_g2 h2 + b2) * feed_forward(h2)

so everything between two residual updates hangs on two input projections (queries / keys / values / gate of the
mixer; gate / up / gate of the feed-forward) and two output projections, and one kernel per layer sums the
gated branches, applies what precedes a repeated pass of a looped block and norms the result twice
(`ops.gated_residual`).  The model plugs into the same engine, paged cache and decode graph as `TransformerLM`.

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
from ..ops import MapsSpec, Proj
from ..ops.mixers import hgrn2_state_shape
from ..parallel.comm import TPGroup
from .config import LayerSpec, ModelConfig, RopeSpec, rope_frequencies
from .kv_cache import KVLayer, PagedKVCache, StateLayer
from .transformer import pick_splits

SMALL_BATCH = 128


class HybridLayer:
    """Device weights of one layer, input projections stacked: w_in1 = [mixer inputs; gate 1], w_in2 = [gate; up; gate 2]."""

    def __init__(self, cfg: ModelConfig, spec: LayerSpec, index: int, get, dtype: torch.dtype):
        p = f"l{index}."
        m = spec.mixer
        f32 = lambda name: get(name).float().contiguous()
        mat = lambda *names: torch.cat([get(n).to(dtype) for n in names]).contiguous()
        self.spec = spec
        self.norms = [f32(p + "norm1")] + ([f32(p + "norm2")] if spec.ff else [])
        if m.kind == "hgrn2":
            self.w_in1 = mat(p + "mix.q", p + "mix.f", p + "mix.v", p + "rg1")
            self.widths = [m.heads * m.dim, m.heads * m.dim, m.heads * m.vdim]
            self.f_bias, self.lower, self.head_norm = f32(p + "mix.f.b"), f32(p + "mix.lower"), f32(p + "mix.norm")
        else:
            self.w_in1 = mat(p + "mix.q", p + "mix.k", p + "mix.v", p + "rg1")
            self.widths = [m.heads * 2 * m.dim, m.kv_heads * 2 * m.dim, m.kv_heads * m.vdim]
            dot = lambda a, b: float(torch.exp((get(p + "mix." + a).double() * get(p + "mix." + b).double()).sum()))
            lam = dot("lq1", "lk1") - dot("lq2", "lk2") + m.diff
            self.maps = MapsSpec(m.heads, m.kv_heads, m.dim, m.vdim, m.scale, maps=2, softcap=m.softcap, lam=lam,
                                 out_scale=1.0 - m.diff, eps=cfg.rms_eps, tiled=dtype == torch.bfloat16)
        self.w_o = mat(p + "mix.o")
        self.gate_bias = [f32(p + "rg1.b")]
        if spec.ff:
            self.w_in2 = mat(p + "mlp.gate", p + "mlp.up", p + "rg2")
            self.w_down = mat(p + "mlp.down")
            self.gate_bias.append(f32(p + "rg2.b"))
        if sum(self.widths) + cfg.hidden_size != self.w_in1.shape[0]:
            raise ValueError(f"layer {index}: projection sizes do not fit the configuration")

    def cache_layer(self):
        m = self.spec.mixer
        if m.kind == "hgrn2":
            return StateLayer(hgrn2_state_shape(m.heads, m.dim, m.vdim))
        return KVLayer(m.kv_heads, self.maps.maps * self.maps.dim_p, self.maps.vdim_p)


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
        self.head = get("head").to(dtype).contiguous()
        self.final_norm = get("final.norm").float().contiguous()
        self.layers: List[HybridLayer] = [HybridLayer(cfg, s, i, get, dtype) for i, s in enumerate(cfg.layers)]
        self.runs = cfg.layer_runs()
        self.loop_step = get("loop.step").float().contiguous() if cfg.loop else None
        self._rope: Dict[RopeSpec, torch.Tensor] = {}

    # ------------------------------------------------------------------ cache
    def new_cache(self, num_blocks: int, max_batch: int, max_seq_len: int,
                  enable_prefix_sharing: bool = True) -> PagedKVCache:
        max_blocks = (max_seq_len + self.cfg.block_size - 1) // self.cfg.block_size
        self._extend_rope(max_blocks * self.cfg.block_size)
        return PagedKVCache.for_layers([self.layers[i].cache_layer() for i, _ in self.runs], num_blocks, max_batch,
                                       max_blocks, self.device, self.dtype, enable_prefix_sharing)

    def _extend_rope(self, positions: int) -> None:
        """cos / sin tables [positions, dims] of every rotation the layers use."""
        for layer in self.layers:
            if layer.spec.mixer.kind != "attention":
                continue
            rope = layer.spec.mixer.rope
            if rope not in self._rope or self._rope[rope].shape[0] < positions:
                freq, mult = rope_frequencies(rope)
                self._rope[rope] = ops.rope_table(rope.dims, positions, inv_freq=freq, scaling=mult, device=self.device)

    def weight_bytes(self) -> int:
        ts = [self.embed, self.head]
        for l in self.layers:
            ts += [l.w_in1, l.w_o] + ([l.w_in2, l.w_down] if l.spec.ff else [])
        return sum(t.numel() * t.element_size() for t in ts)

    # ------------------------------------------------------------------ layers
    def _project(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """fp32 (split-K partials) for small batches, bf16 for large ones, fp32 for 32-bit models."""
        if x.dtype == torch.float32:
            return ops.linear(x, w)
        if x.shape[0] <= SMALL_BATCH:
            splits = pick_splits(w.shape[0], w.shape[1])
            return ops.linear(x, w, splits=splits) if splits > 1 else ops.linear(x, w, fp32_out=True)
        return ops.linear(x, w, swap=False)

    def _feed_forward(self, layer: HybridLayer, h: torch.Tensor):
        """(down projection, gate slice) of the feed-forward branch."""
        ff, width = layer.spec.ff, self.cfg.hidden_size
        if x_small(h):
            y = self._project(h, layer.w_in2)
            act = ops.gated_act(Proj(y, 0, ff), Proj(y, ff, ff), layer.spec.act, dtype=h.dtype)
            gate = Proj(y, 2 * ff, width)
        else:
            act = ops.linear(h, layer.w_in2[:2 * ff], gated=True, act=layer.spec.act, swap=False)
            gate = Proj(ops.linear(h, layer.w_in2[2 * ff:], swap=False), 0, width)
        return Proj(self._project(act, layer.w_down), 0, width), gate

    def _mixer(self, layer: HybridLayer, y: torch.Tensor, run: int, cache: PagedKVCache, b: "Batch") -> torch.Tensor:
        m = layer.spec.mixer
        c1, c2 = layer.widths[0], layer.widths[0] + layer.widths[1]
        first, second, third = Proj(y, 0, c1), Proj(y, c1, layer.widths[1]), Proj(y, c2, layer.widths[2])
        if m.kind == "hgrn2":
            return ops.hgrn2(first, second, third, layer.f_bias, layer.lower, layer.head_norm, cache.state[run],
                             b.context_lens, heads=m.heads, dim=m.dim, vdim=m.vdim, eps=self.cfg.rms_eps,
                             q_start=b.q_start, q_lens=b.q_lens, rows=b.rows, dtype=self.dtype)
        q = ops.maps_append(layer.maps, first, second, third, self._rope[m.rope], b.positions, b.slots, cache.k[run],
                            cache.v[run])
        return ops.maps_attention(layer.maps, q, cache.k[run], cache.v[run], b.block_table, b.context_lens,
                                  q_start=b.q_start, q_lens=b.q_lens, max_q_len=b.max_q_len)

    def _forward(self, ids: torch.Tensor, cache: PagedKVCache, b: "Batch", return_hidden: bool = False):
        cfg, width = self.cfg, self.cfg.hidden_size
        norm = dict(groups=cfg.norm_groups, eps=cfg.rms_eps, dtype=self.dtype)
        start = cfg.loop.start if cfg.loop else -1

        def ahead(r):
            """What is added to the residual before run r, and the norms that read it."""
            if r == len(self.runs):
                return dict(norms=[self.final_norm])
            i, t = self.runs[r]
            pre = dict(norms=self.layers[i].norms)
            if t >= 0 and i == start:
                pre["add_row"] = self.loop_step[t]
                if t > 0:
                    pre["add_mat"] = embedded
            return pre

        first = ahead(0)
        x, h = ops.gated_residual(None, ids=ids, table=self.embed, scale=cfg.embedding_scale,
                                  norms=[] if "add_row" in first else first["norms"], **norm)
        embedded = x
        if "add_row" in first:
            x, h = ops.gated_residual(x, **first, **norm)
        taps = []
        for r, (i, _) in enumerate(self.runs):
            layer = self.layers[i]
            y1 = self._project(h[0], layer.w_in1)
            mixed = self._mixer(layer, y1, r, cache, b)
            branches = [(Proj(self._project(mixed, layer.w_o), 0, width), Proj(y1, sum(layer.widths), width),
                         layer.gate_bias[0])]
            if layer.spec.ff:
                branches.append((*self._feed_forward(layer, h[1]), layer.gate_bias[1]))
            if return_hidden:
                taps.append(ops.gated_residual(x, branches)[0])
            x, h = ops.gated_residual(x, branches, **ahead(r + 1), **norm)
        return (h[0], taps) if return_hidden else h[0]

    # ------------------------------------------------------------------ the engine's entry points
    def prefill(self, ids, positions, slots, cache, block_table, q_start, q_lens, context_lens, max_q_len,
                return_hidden: bool = False, rows: Optional[torch.Tensor] = None):
        """Packed step over the new tokens of several sequences (whole prompts, portions of prompts, single tokens);
        rows[b] is the batch row (state slot) of sequence b.  Returns the final-normed hidden states [T, W] (and the
        residual stream after every layer run)."""
        return self._forward(ids, cache, Batch(positions, slots, block_table, context_lens, q_start, q_lens, max_q_len,
                                               rows), return_hidden)

    def decode_step(self, ids, positions, slots, cache, block_table, context_lens, return_hidden: bool = False):
        """One new token for every batch row; rows with a negative context length are inactive."""
        return self._forward(ids, cache, Batch(positions, slots, block_table, context_lens), return_hidden)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits [rows, vocab]."""
        return ops.linear(hidden, self.head, fp32_out=True)

    def greedy(self, hidden: torch.Tensor, out_ids: Optional[torch.Tensor] = None) -> torch.Tensor:
        return ops.argmax(self.logits(hidden), out_ids=out_ids)

    def close(self) -> None:
        pass


class Batch:
    """Where the tokens of a step sit: cache slots, block tables, and how they are grouped into sequences (q_lens
    None: one per batch row)."""
    __slots__ = ("positions", "slots", "block_table", "context_lens", "q_start", "q_lens", "max_q_len", "rows")

    def __init__(self, positions, slots, block_table, context_lens, q_start=None, q_lens=None, max_q_len=1, rows=None):
        self.positions, self.slots, self.block_table, self.context_lens = positions, slots, block_table, context_lens
        self.q_start, self.q_lens, self.max_q_len, self.rows = q_start, q_lens, max_q_len, rows


def x_small(h: torch.Tensor) -> bool:
    """Whether the feed-forward's input projection leaves its activation to a kernel of its own."""
    return h.dtype == torch.float32 or h.shape[0] <= SMALL_BATCH
