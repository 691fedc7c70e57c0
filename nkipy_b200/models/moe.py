"""Mixture-of-experts FFN block with expert parallelism.

The reference keeps every expert on every rank and shards the expert intermediate
dimension (tensor parallelism), evaluating experts with per-token loops or batched
gathers (examples/models/qwen3/kernels/transformer_layer.py:70-115,
examples/models/gpt_oss/kernels/feedforward.py:39-206).  Here the default is expert
parallelism: rank r owns experts [r * E / ep, (r + 1) * E / ep); activations are
replicated by the preceding tensor-parallel reduction, so *dispatch* is a local
sort-and-gather of the pairs routed to local experts, the experts run as two grouped
tcgen05 GEMMs (SwiGLU fused into the first), and *combine* sums the weighted expert
outputs per token locally and then over ranks.  `moe_parallel="tp"` reproduces the
reference's sharding with the same code path (all experts local, narrower experts).
"""

from __future__ import annotations

from typing import List, Optional

import torch

from .. import ops
from ..ops import Branch, Proj
from ..parallel.comm import TPGroup
from .config import ModelConfig


class MoEBlock:
    def __init__(self, cfg: ModelConfig, tp: TPGroup, moe_parallel: str = "ep"):
        self.cfg, self.tp, self.mode = cfg, tp, moe_parallel
        if moe_parallel == "ep" and cfg.num_experts % tp.world_size:
            raise ValueError("expert parallelism needs num_experts divisible by the number of ranks")
        self.num_local = cfg.num_experts // tp.world_size if moe_parallel == "ep" else cfg.num_experts
        self.expert_lo = tp.rank * self.num_local if moe_parallel == "ep" else 0

    def route(self, lw, x: torch.Tensor):
        logits = ops.linear(x, lw.router, splits=route_splits(x.shape[1]))
        return ops.router_topk(logits, self.cfg.top_k, self.cfg.router_mode, bias=lw.router_bias)

    def _experts(self, lw, x: torch.Tensor):
        """Route, dispatch and run the local experts; returns (y_sorted, plan, routing weights)."""
        cfg = self.cfg
        T = x.shape[0]
        weights, experts = self.route(lw, x)
        plan = ops.moe_dispatch(x, experts, self.expert_lo, self.num_local)
        h = ops.grouped_linear(plan.x_sorted, lw.gate_up, plan.offsets, max_rows_per_group=T, gated=True,
                               bias=lw.gate_up_bias, act_limit=cfg.swiglu_limit, act_alpha=cfg.swiglu_alpha,
                               tiles=plan.tiles)
        y_sorted = ops.grouped_linear(h, lw.down, plan.offsets, max_rows_per_group=T, bias=lw.down_bias,
                                      tiles=plan.tiles)
        return y_sorted, plan, weights

    def forward(self, lw, x: torch.Tensor) -> torch.Tensor:
        """x [T, H] (normed hidden states, replicated over ranks) -> MoE output [T, H], summed over ranks."""
        y_sorted, plan, weights = self._experts(lw, x)
        y = ops.moe_combine(y_sorted, plan.pair_pos, weights, x.shape[0])
        self.tp.all_reduce(y)
        return y

    def forward_add_rmsnorm(self, lw, x: torch.Tensor, resid: torch.Tensor, next_norm: torch.Tensor):
        """MoE block + residual + next RMSNorm; returns (new residual, normed).  With the fused
        tensor-parallel runtime the combine kernel pushes its partial rows straight into the peers'
        buffers and the reducing norm kernel sums them (no library collective)."""
        cfg = self.cfg
        fused = getattr(self.tp, "fused", None)
        T = x.shape[0]
        if fused is not None and T <= fused.max_tokens:
            y_sorted, plan, weights = self._experts(lw, x)
            return fused.moe_combine_allreduce_add_rmsnorm(y_sorted, plan.pair_pos, weights, T, resid, next_norm,
                                                           cfg.rms_eps)
        y = self.forward(lw, x)
        return ops.add_rmsnorm(y, next_norm, residual_in=resid, eps=cfg.rms_eps)

    def forward_sharded(self, lw, x_local: torch.Tensor) -> torch.Tensor:
        """Expert-parallel block for tokens that are sharded over the ranks (x_local [T / ranks, H], this rank's
        slab): the rows travel to their experts' owners and back through peer memory
        (`parallel.moe_a2a.MoEAllToAll`).  Returns this rank's slab of the block output."""
        from ..parallel.moe_a2a import MoEAllToAll

        cfg = self.cfg
        T = x_local.shape[0]
        a2a = getattr(self, "_a2a", None)
        if a2a is None or a2a.max_local_tokens < T:
            if a2a is not None:
                a2a.close()
            cap = max(2048, 1 << (T - 1).bit_length())
            a2a = self._a2a = MoEAllToAll(self.tp, cap, cfg.top_k, cfg.hidden_size, cfg.num_experts)
        weights, experts = self.route(lw, x_local)
        return a2a.forward(x_local, experts, weights, lw.gate_up, lw.down, gate_up_bias=lw.gate_up_bias,
                           down_bias=lw.down_bias, act_limit=cfg.swiglu_limit, act_alpha=cfg.swiglu_alpha)


def route_splits(width: int, tokens: int = 1) -> int:
    """Split-K factor of a router's product: its few outputs are one weight tile, so several SMs share the contraction of a
    row tile when there are few of those."""
    return max(2, min(16, width // 256, 296 // max(tokens // 128, 1)))


class RoutedExperts:
    """Routed feed-forward of one layer of a layer-by-layer decoder (`config.ExpertsSpec`, one rank).  The (weighted) sum of
    the experts' rows is left to the residual kernel (`ops.Branch`).  bf16 sizes with 16-byte rows run the grouped
    tcgen05 products, everything else the grouped products on the CUDA cores.

    Rows for the input projection of a layer whose sublayers share their input: `w_wide` the shared expert's [gate; up] (None
    without one), `w_narrow` [router; shared gate]."""

    def __init__(self, spec, t):
        self.spec = spec
        self.gate_up = torch.stack([t.mat(f"e{e}.gate", f"e{e}.up") for e in range(spec.experts)]).contiguous()
        self.down = t.stack(*[f"e{e}.down" for e in range(spec.experts)])
        self.tiled = t.dtype == torch.bfloat16 and self.down.shape[1] % 8 == 0 and spec.ff % 8 == 0
        self.w_wide, self.shared_down = None, None
        self.w_narrow = t.mat("router")
        if spec.shared:
            self.w_wide, self.shared_down = t.mat("shared.gate", "shared.up"), t.mat("shared.down")
            self.w_narrow = t.mat("router", "shared.sg")

    def weights(self):
        return [w for w in (self.w_narrow, self.gate_up, self.down, self.w_wide, self.shared_down) if w is not None]

    def run(self, model, h: torch.Tensor, wide: Optional[Proj] = None, narrow: Optional[Proj] = None) -> List[Branch]:
        """wide / narrow: results of `w_wide` and `w_narrow` when the layer has them already."""
        s, (T, W) = self.spec, h.shape
        if narrow is None:
            z = ops.linear(h, self.w_narrow, splits=route_splits(W, T)) if h.dtype == torch.bfloat16 else ops.linear(h, self.w_narrow)
            narrow = Proj(z, 0, self.w_narrow.shape[0])
        logits = Proj(narrow.t, narrow.col, s.experts)
        if s.score == "sigmoid":
            weights, experts = ops.router_topk(logits, s.top, "sigmoid_topk", scale=s.scale)
        else:
            weights, experts = ops.router_topk(logits, s.top, groups=s.groups, keep=s.keep, scale=s.scale)
        gather = self.tiled or s.scale_input
        plan = ops.moe_dispatch(h, experts, 0, s.experts, gather=gather, weights=weights if s.scale_input else None)
        if self.tiled:
            act = ops.grouped_linear(plan.x_sorted, self.gate_up, plan.offsets, max_rows_per_group=T, gated=True,
                                     act_limit=s.limit, tiles=plan.tiles)
            y = ops.grouped_linear(act, self.down, plan.offsets, max_rows_per_group=T, tiles=plan.tiles)
        else:
            gu = ops.grouped_linear_simt(plan, plan.x_sorted, self.gate_up, gather)
            act = ops.gated_act(Proj(gu, 0, s.ff), Proj(gu, s.ff, s.ff), "clamped" if s.limit else "silu", dtype=h.dtype,
                                limit=s.limit)
            y = ops.grouped_linear_simt(plan, act, self.down, True)
        if s.scale_input:
            out = [Branch(Proj(y, 0, W), pair_pos=plan.pair_pos, top_k=s.top)]
        else:
            out = [Branch(Proj(y, 0, W), pair_pos=plan.pair_pos, pair_w=weights)]
        if s.shared:
            n, limit = s.shared.ff, s.shared.limit
            if wide is None:
                wide = Proj(model.project(h, self.w_wide), 0, 2 * n)
            act = ops.gated_act(Proj(wide.t, wide.col, n), Proj(wide.t, wide.col + n, n), "clamped", dtype=h.dtype, limit=limit)
            out.append(Branch(Proj(model.project(act, self.shared_down), 0, W), Proj(narrow.t, narrow.col + s.experts, 1)))
        return out
