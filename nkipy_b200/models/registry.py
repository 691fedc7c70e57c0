"""Model folders -> models: the architecture named in config.json picks the configuration reader, the weight reader
and the model class.

A folder holds config.json and the weights, either as a checkpoint (``*.safetensors`` under the architecture's own
tensor names) or as prepared per-rank shards (``shard_{rank}.safetensors``, see `checkpoint.prepare_checkpoint`).
"""

from __future__ import annotations

import glob
import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, Optional

import torch

from . import config as C
from .checkpoint import LazyCheckpoint, convert_state_dict
from .hybrid import HybridLM
from .transformer import TransformerLM
from .weights import hybrid_random_weights, load_shard, random_weights

# Hugging Face field -> ModelConfig field
_HF_FIELDS = {"vocab_size": "vocab_size", "hidden_size": "hidden_size", "num_hidden_layers": "num_layers",
              "num_attention_heads": "num_heads", "num_key_value_heads": "num_kv_heads", "head_dim": "head_dim",
              "intermediate_size": "intermediate_size", "rms_norm_eps": "rms_eps", "rope_theta": "rope_theta"}


def _hf_config(preset: Callable[..., C.ModelConfig], **fields: str):
    """Reader of a Hugging Face config.json on top of a preset; `fields` adds to or replaces `_HF_FIELDS`."""
    names = {**_HF_FIELDS, **fields}

    def read(raw: dict) -> C.ModelConfig:
        cfg = preset(**({"num_layers": raw["num_hidden_layers"]} if "num_hidden_layers" in raw else {}))
        for src, dst in names.items():
            if dst and raw.get(src) is not None:
                setattr(cfg, dst, raw[src])
        if "head_dim" not in raw and "num_attention_heads" in raw and "hidden_size" in raw:
            cfg.head_dim = raw["hidden_size"] // raw["num_attention_heads"]
        return cfg

    return read


@dataclass(frozen=True)
class Architecture:
    config: Callable[[dict], C.ModelConfig]
    model: type
    read: Callable                        # (cfg, LazyCheckpoint, rank, world, moe_parallel) -> weights
    random: Callable                      # (cfg, rank, world, device, seed, moe_parallel) -> weights


def _transformer(config) -> Architecture:
    return Architecture(
        config, TransformerLM,
        lambda cfg, sd, rank, world, moe: convert_state_dict(cfg, sd, rank, world, moe),
        lambda cfg, rank, world, device, seed, moe: random_weights(cfg, rank, world, device=device, seed=seed,
                                                                   moe_parallel=moe))


def _hybrid(config) -> Architecture:
    return Architecture(
        config, HybridLM,
        lambda cfg, sd, rank, world, moe: {k: sd[k] for k in sd.keys()},
        lambda cfg, rank, world, device, seed, moe: hybrid_random_weights(cfg, device=device, seed=seed))


_MOE = {"num_experts_per_tok": "top_k", "intermediate_size": ""}

ARCHITECTURES: Dict[str, Architecture] = {
    "LlamaForCausalLM": _transformer(_hf_config(C.llama3_8b)),
    "Qwen3ForCausalLM": _transformer(_hf_config(lambda **kw: C.qwen3_embedding("0.6b", **kw))),
    "Qwen3MoeForCausalLM": _transformer(_hf_config(C.qwen3_30b_a3b, **_MOE, num_experts="num_experts",
                                                   moe_intermediate_size="moe_intermediate_size")),
    "GptOssForCausalLM": _transformer(_hf_config(C.gpt_oss_20b, **{**_MOE, "intermediate_size": "moe_intermediate_size"},
                                                 num_local_experts="num_experts", sliding_window="sliding_window")),
    "Tolenex": _hybrid(C.tolenex_config),
    "Mumilorn": _hybrid(C.mumilorn_config),
    "Ligizen": _hybrid(C.ligizen_config),
    "Redodra": _hybrid(C.redodra_config),
}


def architecture_of(raw: dict) -> Architecture:
    name = raw.get("architecture") or (raw.get("architectures") or [None])[0]
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(ARCHITECTURES))}")
    return ARCHITECTURES[name]


def for_config(cfg: C.ModelConfig) -> Architecture:
    """The architecture entry that runs a configuration made in code."""
    if cfg.layers is None:
        return ARCHITECTURES["LlamaForCausalLM"]
    return ARCHITECTURES[{"mumilorn": "Mumilorn", "ligizen": "Ligizen", "redodra": "Redodra"}.get(cfg.name, "Tolenex")]


def read_config(folder: str):
    """(architecture, configuration) of a model folder."""
    with open(os.path.join(folder, "config.json")) as f:
        raw = json.load(f)
    arch = architecture_of(raw)
    return arch, arch.config(raw)


def build(arch: Architecture, cfg: C.ModelConfig, weights, tp=None, device=None, dtype: torch.dtype = torch.bfloat16,
          moe_parallel: str = "ep"):
    if arch.model is TransformerLM:
        if dtype != torch.bfloat16:
            raise ValueError(f"{cfg.name} runs in bfloat16")
        return TransformerLM(cfg, weights, tp, device=device, moe_parallel=moe_parallel)
    return arch.model(cfg, weights, tp, device=device, dtype=dtype)


def load_model(folder: str, tp=None, device=None, dtype: torch.dtype = torch.bfloat16, moe_parallel: str = "ep",
               weights_folder: Optional[str] = None):
    """Model of a folder on `device`; weights_folder overrides where the weights lie."""
    arch, cfg = read_config(folder)
    rank, world = (tp.rank, tp.world_size) if tp is not None else (0, 1)
    src = weights_folder or folder
    if glob.glob(os.path.join(src, f"shard_{rank}.safetensors")):
        weights = load_shard(src, rank, device=device or "cpu")
    else:
        weights = arch.read(cfg, LazyCheckpoint(src), rank, world, moe_parallel)
    return build(arch, cfg, weights, tp, device, dtype, moe_parallel)
