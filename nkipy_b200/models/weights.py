"""Weight preparation: per-rank shards in the reference's safetensors schema.

Key names and orientation follow the reference converters
(examples/models/qwen3/tensor_preparation.py:126-248,
examples/models/qwen3_embedding/prepare_weights.py:37-76): every matrix is
stored in ``x @ W`` orientation,

    tok_embedding [V, H]            norm_weight [H]         lm_head_weight [H, V/tp]
    layers.{i}.qkv_weight [H, (nq + 2 nkv) d / tp]          layers.{i}.o_weight [nq d / tp, H]
    layers.{i}.input_layernorm_weight [H]                   layers.{i}.post_attention_layernorm_weight [H]
    dense:  layers.{i}.gate_up_weight [H, 2 I / tp]  (gate | up)   layers.{i}.down_weight [I / tp, H]
    MoE:    layers.{i}.router_weight [H, E]
            layers.{i}.gate_up_weight [E_local, H, 2 I_local]      layers.{i}.down_weight [E_local, I_local, H]
    Qwen3:  layers.{i}.q_norm_weight [d], k_norm_weight [d]
    gpt-oss: qkv_bias, o_bias, router_bias, gate_up_bias, down_bias, sinks [nq / tp]

Column-parallel tensors (qkv, gate_up, lm_head) are split on their output axis,
row-parallel ones (o, down) on their input axis; KV heads are replicated when a
rank would own less than one head (tensor_preparation.py:82-91).  The reference
shards MoE experts on the intermediate axis (every rank holds all experts);
`moe_parallel="ep"` shards the expert axis instead (new here).
"""

from __future__ import annotations

import os
from typing import Dict, Optional

import torch

from .config import ModelConfig


def _normal(shape, std, seed, device, dtype=torch.bfloat16):
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    return (torch.randn(shape, generator=g, device=device, dtype=torch.float32) * std).to(dtype)


def kv_heads_for_rank(cfg: ModelConfig, rank: int, world: int):
    """(first kv head, number of kv heads) owned by `rank`; heads are replicated when world > num_kv_heads."""
    if cfg.num_kv_heads >= world:
        n = cfg.num_kv_heads // world
        return rank * n, n
    rep = world // cfg.num_kv_heads
    return rank // rep, 1


def shard_qkv(w_q, w_k, w_v, cfg: ModelConfig, rank: int, world: int):
    """Fuse this rank's q / k / v columns: [H, (nq_l + 2 nkv_l) d]."""
    d = cfg.head_dim
    nq_l = cfg.num_heads // world
    kv0, nkv_l = kv_heads_for_rank(cfg, rank, world)
    q = w_q[..., rank * nq_l * d:(rank + 1) * nq_l * d]
    k = w_k[..., kv0 * d:(kv0 + nkv_l) * d]
    v = w_v[..., kv0 * d:(kv0 + nkv_l) * d]
    return torch.cat([q, k, v], dim=-1).contiguous()


def random_weights(cfg: ModelConfig, rank: int = 0, world: int = 1, device="cpu", seed: int = 0, std: float = 0.02,
                   moe_parallel: str = "ep", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random-init weights ~ N(0, std) for `rank` of `world`, in the schema above.  The
    full tensor of every parameter is generated from a per-parameter seed and then
    sliced, so all ranks of any world size see shards of the same model."""
    H, d, V = cfg.hidden_size, cfg.head_dim, cfg.vocab_size
    out: Dict[str, torch.Tensor] = {}
    sid = [seed * 100003]

    def nxt():
        sid[0] += 1
        return sid[0]

    out["tok_embedding"] = _normal((V, H), std, nxt(), device, dtype)
    out["norm_weight"] = torch.ones(H, dtype=dtype, device=device)
    v_l = V // world
    lm = _normal((H, V), std, nxt(), device, dtype)
    out["lm_head_weight"] = lm[:, rank * v_l:(rank + 1) * v_l].contiguous()
    del lm
    for i in range(cfg.num_layers):
        p = f"layers.{i}."
        wq = _normal((H, cfg.q_size), std, nxt(), device, dtype)
        wk = _normal((H, cfg.kv_size), std, nxt(), device, dtype)
        wv = _normal((H, cfg.kv_size), std, nxt(), device, dtype)
        out[p + "qkv_weight"] = shard_qkv(wq, wk, wv, cfg, rank, world)
        del wq, wk, wv
        nq_l = cfg.num_heads // world
        wo = _normal((cfg.q_size, H), std, nxt(), device, dtype)
        out[p + "o_weight"] = wo[rank * nq_l * d:(rank + 1) * nq_l * d].contiguous()
        del wo
        out[p + "input_layernorm_weight"] = torch.ones(H, dtype=dtype, device=device)
        out[p + "post_attention_layernorm_weight"] = torch.ones(H, dtype=dtype, device=device)
        if cfg.qk_norm:
            out[p + "q_norm_weight"] = torch.ones(d, dtype=dtype, device=device)
            out[p + "k_norm_weight"] = torch.ones(d, dtype=dtype, device=device)
        if cfg.attn_bias:
            bq = _normal((cfg.q_size,), std, nxt(), device, dtype)
            bk = _normal((cfg.kv_size,), std, nxt(), device, dtype)
            bv = _normal((cfg.kv_size,), std, nxt(), device, dtype)
            out[p + "qkv_bias"] = shard_qkv(bq, bk, bv, cfg, rank, world)
            bo = _normal((H,), std, nxt(), device, dtype)
            # row-parallel bias is applied once: only rank 0 keeps it (gpt_oss/tensor_preparation.py:131-133)
            out[p + "o_bias"] = bo if rank == 0 else torch.zeros_like(bo)
        if cfg.attention_sinks:
            s = _normal((cfg.num_heads,), 1.0, nxt(), device, torch.float32)
            out[p + "sinks"] = s[rank * nq_l:(rank + 1) * nq_l].contiguous()
        if not cfg.is_moe:
            I = cfg.intermediate_size
            i_l = I // world
            wg = _normal((H, I), std, nxt(), device, dtype)
            wu = _normal((H, I), std, nxt(), device, dtype)
            out[p + "gate_up_weight"] = torch.cat(
                [wg[:, rank * i_l:(rank + 1) * i_l], wu[:, rank * i_l:(rank + 1) * i_l]], dim=-1).contiguous()
            del wg, wu
            wd = _normal((I, H), std, nxt(), device, dtype)
            out[p + "down_weight"] = wd[rank * i_l:(rank + 1) * i_l].contiguous()
            del wd
        else:
            E, I = cfg.num_experts, cfg.moe_intermediate_size
            out[p + "router_weight"] = _normal((H, E), std, nxt(), device, dtype)
            if cfg.router_bias:
                out[p + "router_bias"] = _normal((E,), std, nxt(), device, dtype)
            if moe_parallel == "ep":
                e_l, i_l = E // world, I
                e0, i0 = rank * e_l, 0
            else:
                e_l, i_l = E, I // world
                e0, i0 = 0, rank * i_l
            gs, us, ds = nxt(), nxt(), nxt()
            gu = torch.empty((e_l, H, 2 * i_l), dtype=dtype, device=device)
            dn = torch.empty((e_l, i_l, H), dtype=dtype, device=device)
            for e in range(e_l):
                ge = e0 + e
                wg = _normal((H, I), std, gs * 1009 + ge, device, dtype)
                wu = _normal((H, I), std, us * 1009 + ge, device, dtype)
                wd = _normal((I, H), std, ds * 1009 + ge, device, dtype)
                gu[e, :, :i_l] = wg[:, i0:i0 + i_l]
                gu[e, :, i_l:] = wu[:, i0:i0 + i_l]
                dn[e] = wd[i0:i0 + i_l]
            out[p + "gate_up_weight"] = gu
            out[p + "down_weight"] = dn
            if cfg.expert_bias:
                bgs, bds = nxt(), nxt()
                bgu = torch.empty((e_l, 2 * i_l), dtype=dtype, device=device)
                bd = torch.empty((e_l, H), dtype=dtype, device=device)
                for e in range(e_l):
                    ge = e0 + e
                    b = _normal((2 * I,), std, bgs * 1009 + ge, device, dtype)
                    bgu[e, :i_l] = b[i0:i0 + i_l]
                    bgu[e, i_l:] = b[I + i0:I + i0 + i_l]
                    b2 = _normal((H,), std, bds * 1009 + ge, device, dtype)
                    bd[e] = b2 if (moe_parallel == "ep" or rank == 0) else torch.zeros_like(b2)
                out[p + "gate_up_bias"] = bgu
                out[p + "down_bias"] = bd
    return out


def _mixer_shapes(m, W: int) -> Dict[str, tuple]:
    """Tensors of a token mixer (models/mixers.py) by their names under '<layer>.mix.'."""
    if m.kind in ("parallel", "blend"):
        out = {"left.out": (W,), "right.out": (W,)} if m.kind == "blend" else {}
        return {**{"left." + k: v for k, v in _mixer_shapes(m.left, W).items()},
                **{"right." + k: v for k, v in _mixer_shapes(m.right, W).items()}, **out}
    if m.kind == "rwkv":
        c, rank = m.heads * m.dim, m.rank or 16
        return {**{f"mu.{n}": (W,) for n in "rkvgw"}, **{n: (c, W) for n in "rkvg"}, "w1": (rank, W), "w2": (c, rank),
                "w0": (c,), "u": (m.heads, m.dim), "norm": (c,), "o": (W, c)}
    out = m.heads * m.vdim
    if m.kind == "ssd":
        channels = out + 2 * m.groups * m.state
        return {"in": (out + channels + m.heads, W), "conv": (channels, m.conv), "conv.b": (channels,), "dt_bias": (m.heads,),
                "A_log": (m.heads,), "D": (m.heads,), "norm": (out,), "o": (W, out)}
    if m.kind == "delta":
        c = m.kv_heads * m.dim
        return {"q": (c, W), "q.conv": (c, m.conv), "k": (c, W), "k.conv": (c, m.conv), "v": (out, W), "v.conv": (out, m.conv),
                "b": (m.heads, W), "a": (m.heads, W), "A_log": (m.heads,), "dt_bias": (m.heads,), "norm": (m.vdim,),
                "g": (out, W), "o": (W, out)}
    if m.kind == "grouped":
        rows = {"q": m.heads * m.dim}
        if m.kv_from is None:
            rows.update(k=m.kv_heads * m.dim, v=m.kv_heads * m.vdim)
        shapes = {**{k: (n, W) for k, n in rows.items()}, "o": (W, out)}
        if m.bias:
            shapes.update({k + ".b": (n,) for k, n in {**rows, "o": W}.items()})
        per_head = (("r1", "r2") if m.distance else ()) + (("sink",) if m.sink else ())
        return {**shapes, **{k: (m.heads,) for k in per_head}, **({"g": (m.heads, W)} if m.gate else {})}
    if m.kind == "chunk":
        q, k, v = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
        own = {} if m.kv_from is not None else {"k": (k, W), "k.b": (k,), "v": (v, W), "v.b": (v,)}
        return {"q": (q, W), "q.b": (q,), **own, "g": (m.heads, W), "o": (W, out)}
    if m.kind == "latent":
        return {"dq": (m.q_rank, W), "dq.norm": (m.q_rank,), "uq": (m.heads * (m.dim + m.rot), m.q_rank),
                "dkv": (m.kv_rank + m.rot, W), "dkv.norm": (m.kv_rank,), "uk": (m.heads * m.dim, m.kv_rank),
                "uv": (out, m.kv_rank), "sink": (m.heads,), "g": (m.heads, W), "o": (W, out)}
    if m.kind == "window":
        q, k = m.heads * m.dim, m.kv_heads * m.dim
        return {"q": (q, W), "k": (k, W), "v": (m.kv_heads * m.vdim, W), "q.norm": (q,), "k.norm": (k,), "g": (out, W),
                "o": (W, out)}
    if m.kind == "gla":
        c, rank = m.heads * m.dim, m.rank or 16
        return {"q": (c, W), "k": (c, W), "v": (out, W), "g": (out, W), "a1": (rank, W), "a2": (c, rank), "a2.b": (c,),
                "norm": (m.vdim,), "o": (W, out)}
    if m.kind == "hgrn2":
        c = m.heads * m.dim
        return {"q": (c, W), "f": (c, W), "f.b": (c,), "lower": (c,), "v": (out, W), "norm": (m.vdim,), "o": (W, out)}
    return {"q": (2 * m.heads * m.dim, W), "k": (2 * m.kv_heads * m.dim, W), "v": (m.kv_heads * m.vdim, W), "o": (W, out),
            **{n: (m.dim,) for n in ("lq1", "lk1", "lq2", "lk2")}}


def hybrid_weight_shapes(cfg: ModelConfig) -> Dict[str, tuple]:
    """Name -> shape of every tensor of a layer-by-layer configuration (models/hybrid.py), matrices [out, in]."""
    W, V = cfg.hidden_size, cfg.vocab_size
    out: Dict[str, tuple] = {"embed": (V, W), "final.norm": (W,)}
    if not cfg.tie_embeddings:
        out["head"] = (V, W)
    if cfg.loop:
        out["loop.step"] = (cfg.loop.times, W)
    norm = lambda name: {name: (W,), **({name + ".b": (W,)} if cfg.layer_norm or cfg.tanh_norm else {}),
                         **({name + ".alpha": ()} if cfg.tanh_norm else {})}
    out.update(norm("final.norm"))
    if cfg.token_side:
        out["side.embed"] = (V, len(cfg.layers) * cfg.token_side)
    for i, layer in enumerate(cfg.layers):
        shapes = {**norm("norm1"), **{"mix." + k: v for k, v in _mixer_shapes(layer.mixer, W).items()}}
        if layer.block == "sandwich":
            shapes.update(norm("norm1b"))
        if cfg.depth_average:
            shapes["dwa"] = (i + 2,)
        if layer.block == "gated":
            shapes.update({"rg1": (W, W), "rg1.b": (W,)})
        if (layer.ff or layer.experts) and layer.block != "parallel":
            shapes.update(norm("norm2"))
            if layer.block == "sandwich":
                shapes.update(norm("norm2b"))
        if layer.ff:
            shapes.update({"mlp.up": (layer.ff, W), "mlp.down": (W, layer.ff)})
            if layer.act == "xielu":
                shapes["mlp.act"] = (2,)
            if layer.block not in ("pre-norm", "sandwich"):
                shapes["mlp.gate"] = (layer.ff, W)
            if layer.block == "gated":
                shapes.update({"rg2": (W, W), "rg2.b": (W,)})
        if layer.experts:
            x = layer.experts
            shapes["mlp.router"] = (x.experts, W)
            for e in range(x.experts):
                shapes.update({f"mlp.e{e}.gate": (x.ff, W), f"mlp.e{e}.up": (x.ff, W), f"mlp.e{e}.down": (W, x.ff)})
            if x.shared:
                n = x.shared.ff
                shapes.update({"mlp.shared.gate": (n, W), "mlp.shared.up": (n, W), "mlp.shared.down": (W, n),
                               "mlp.shared.sg": (1, W)})
        if cfg.token_side:
            n = cfg.token_side
            shapes.update({"side.gate": (n, W), "side.proj": (W, n), "side.norm": (W,)})
        out.update({f"l{i}." + k: v for k, v in shapes.items()})
    return out


def hybrid_random_weights(cfg: ModelConfig, device="cpu", seed: int = 0, std: float = 0.02,
                          dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random-init weights of a layer-by-layer configuration: N(0, std), norms that multiply by 1, lower bounds of the
    forget gates and mixes of neighbouring tokens uniform in [0, 0.9), slow decays, depth averages near their last term."""
    out: Dict[str, torch.Tensor] = {}
    for n, (name, shape) in enumerate(hybrid_weight_shapes(cfg).items()):
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2", "norm1b", "norm2b") or name == "final.norm":
            out[name] = torch.full(shape, 1.0 - cfg.norm_offset, dtype=dtype, device=device)
        elif leaf in ("norm", "out", "alpha", "D", "r1"):
            out[name] = torch.ones(shape, dtype=dtype, device=device)
        elif leaf == "r2":
            out[name] = torch.full(shape, 0.1, dtype=dtype, device=device)
        elif leaf == "conv":
            out[name] = _normal(shape, shape[1] ** -0.5, seed * 100003 + n, device, dtype)
        elif leaf == "lower" or ".mu." in name:
            g = torch.Generator(device=device).manual_seed(seed * 100003 + n)
            out[name] = (0.9 * torch.rand(shape, generator=g, device=device)).to(dtype)
        else:
            out[name] = _normal(shape, std, seed * 100003 + n, device, dtype)
            if leaf == "w0":
                out[name] -= 4.0             # exp(-exp(-4)): a memory of some fifty tokens
            elif leaf in ("A_log", "dt_bias"):
                out[name] -= 2.0
            elif leaf == "dwa":
                out[name][-1] += 1.0
    return out


def save_shard(weights: Dict[str, torch.Tensor], directory: str, rank: int) -> str:
    """Write ``shard_{rank}.safetensors`` (same file naming as the reference converter)."""
    from safetensors.torch import save_file

    os.makedirs(directory, exist_ok=True)
    path = os.path.join(directory, f"shard_{rank}.safetensors")
    save_file({k: v.contiguous().cpu() for k, v in weights.items()}, path)
    return path


def load_shard(directory: str, rank: int, device="cpu") -> Dict[str, torch.Tensor]:
    from safetensors.torch import load_file

    return load_file(os.path.join(directory, f"shard_{rank}.safetensors"), device=str(device))


def to_device_layout(w: torch.Tensor) -> torch.Tensor:
    """``x @ W`` orientation [.., K, N] -> K-major [.., N, K] contiguous (the tcgen05 operand layout)."""
    return w.transpose(-1, -2).contiguous()
