"""Command-line plumbing shared by the example entry points (examples/models/*): weights from prepared
shards or random init, prompts from a tokenizer or synthetic ids, generation through the paged engine
and the timing lines the reference scripts print (examples/models/qwen3/qwen3.py:495-537).

    python -m nkipy_b200.models.runner --model DIR -n 64 --batch 4     # any folder the registry knows (registry.py)
"""

from __future__ import annotations

import argparse
import os
import sys
import time
from typing import List, Optional

import torch

from ..parallel.comm import TPGroup
from .config import ModelConfig, ligizen_shape, mumilorn_shape, redodra_shape, tolenex_shape
from .engine import GenerationEngine, Sampling
from .weights import load_shard


def add_common_args(ap: argparse.ArgumentParser) -> None:
    ap.add_argument("prompt", nargs="?", default=None, help="prompt text (needs --model with a tokenizer)")
    ap.add_argument("--checkpoint", default=None, help="directory with shard_{rank}.safetensors; random init if absent")
    ap.add_argument("--model", default=None, help="Hugging Face model directory (tokenizer / config)")
    ap.add_argument("-n", "--max-new-tokens", type=int, default=64)
    ap.add_argument("--batch", type=int, default=1)
    ap.add_argument("--prompt-len", type=int, default=128, help="synthetic prompt length when no tokenizer is given")
    ap.add_argument("--max-seq-len", type=int, default=4096)
    ap.add_argument("--layers", type=int, default=0, help="override the layer count (quick runs)")
    ap.add_argument("--moe-parallel", choices=["ep", "tp"], default="ep")
    ap.add_argument("--no-graph", action="store_true", help="do not capture the decode step in a CUDA graph")
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    ap.add_argument("--top-k", type=int, default=0, help="0: unrestricted")
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16",
                    help="float32: true 32-bit, for the models that have it")
    ap.add_argument("--tiny", action="store_true",
                    help="shrink the model (hidden 256, vocabulary 2048, <= 8 experts) for quick functional runs")


def load_tokenizer(path: Optional[str]):
    if not path:
        return None
    from transformers import AutoTokenizer

    try:
        return AutoTokenizer.from_pretrained(path)
    except (OSError, ValueError):            # a folder without tokenizer files: synthetic ids
        return None


def build_prompts(args, cfg: ModelConfig, tokenizer) -> List[List[int]]:
    if tokenizer is not None and args.prompt:
        ids = tokenizer(args.prompt)["input_ids"]
        return [list(ids) for _ in range(args.batch)]
    g = torch.Generator().manual_seed(args.seed)
    return torch.randint(0, cfg.vocab_size, (args.batch, args.prompt_len), generator=g).tolist()


def shrink(cfg: ModelConfig) -> ModelConfig:
    """Same architecture features, toy sizes."""
    if cfg.name == "mumilorn":
        routed = any(l.experts for l in cfg.layers)
        return mumilorn_shape(256, layers=len(cfg.layers), heads=4, kv_heads=2, ff=512, vocab=2048, dim=32, window=64, rank=16,
                              **(dict(experts=8, top=2, expert_ff=64, groups=4, keep=2) if routed else {}))
    if cfg.name == "ligizen":
        routed = any(l.experts for l in cfg.layers)
        return ligizen_shape(256, layers=len(cfg.layers), heads=4, kv_heads=2, ff=512, vocab=2048, dim=32, window=64, chunk=48,
                             latent_dim=40, rot=8, kv_rank=48, q_rank=96, side=32, share_every=2,
                             **(dict(experts=8, top=2, expert_ff=64) if routed else {}))
    if cfg.name == "redodra":
        return redodra_shape(256, layers=len(cfg.layers), heads=4, kv_heads=2, ff=512, vocab=2048, dim=32, window=64, keep_first=3,
                             state=16, groups=2, share_every=2)
    if cfg.layers is not None:
        return tolenex_shape(256, layers=len(cfg.layers), heads=4, kv_heads=1, ff=512, vocab=2048, dim=32, vdim=64,
                             groups=cfg.norm_groups, loop=cfg.loop, embedding_scale=cfg.embedding_scale)
    over = dict(vocab_size=2048, hidden_size=256, num_heads=4, num_kv_heads=2, head_dim=64, intermediate_size=512,
                max_position=min(cfg.max_position, 4096))
    if cfg.is_moe:
        over.update(num_experts=min(cfg.num_experts, 8), top_k=min(cfg.top_k, 2), moe_intermediate_size=128,
                    intermediate_size=0)
    if cfg.layer_types is not None:
        over["layer_types"] = cfg.layer_types[: max(cfg.num_layers, 1)]
    if cfg.sliding_window:
        over["sliding_window"] = min(cfg.sliding_window, 16)
    return cfg.scaled(**over)


def build_model(cfg: ModelConfig, args, tp: TPGroup, arch=None):
    from . import registry

    if args.layers:
        cfg.num_layers = args.layers
        if cfg.layer_types is not None:
            cfg.layer_types = cfg.layer_types[: args.layers]
        if cfg.layers is not None:
            cfg.layers, cfg.loop = cfg.layers[: args.layers], None
    if getattr(args, "tiny", False):
        cfg = shrink(cfg)
    arch = arch or registry.for_config(cfg)
    if args.checkpoint:
        weights = load_shard(args.checkpoint, tp.rank, device=tp.device)
    else:
        weights = arch.random(cfg, tp.rank, tp.world_size, tp.device, args.seed, args.moe_parallel)
    return registry.build(arch, cfg, weights, tp, tp.device, getattr(torch, args.dtype), args.moe_parallel)


def run_generation(cfg: ModelConfig, args, model=None, tp: Optional[TPGroup] = None) -> int:
    tp = tp or TPGroup.from_env()
    tokenizer = load_tokenizer(args.model)
    if model is None:
        model = build_model(cfg, args, tp)
    prompts = build_prompts(args, model.cfg, tokenizer)
    max_len = min(args.max_seq_len, max(len(p) for p in prompts) + args.max_new_tokens + 64)
    eng = GenerationEngine(model, max_batch=len(prompts), max_seq_len=max_len,
                           use_cuda_graph=not args.no_graph and tp.device.type == "cuda")
    eng.generate([p[:8] for p in prompts], 2)            # warm-up (graph capture, autotuned splits)
    eng.stats.__init__()
    tp.barrier()
    t0 = time.perf_counter()
    out = eng.generate(prompts, args.max_new_tokens,
                       sampling=Sampling(args.temperature, args.top_k, args.top_p, args.seed))
    dt = time.perf_counter() - t0
    if tp.rank == 0:
        s = eng.stats.summary()
        print(f"Time to first token: {s.get('ttft_p50_s', 0.0):.3f}s")
        n = sum(len(o) for o in out)
        print(f"Generated {n} tokens in {dt:.3f}s")
        print(f"Decode tokens/sec: {s.get('decode_tokens_per_s', n / max(dt, 1e-9)):.2f}")
        if tokenizer is not None:
            print(tokenizer.decode(out[0]))
        else:
            print("first sequence ids:", out[0][:32])
    tp.barrier()
    if tp.world_size > 1:
        torch.distributed.destroy_process_group()
    return 0


def main(argv: Optional[List[str]] = None) -> int:
    from . import registry

    ap = argparse.ArgumentParser(description="generate with a model folder (config.json + weights)")
    add_common_args(ap)
    args = ap.parse_args(argv)
    if not args.model:
        ap.error("--model DIR is needed")
    arch, cfg = registry.read_config(args.model)
    tp = TPGroup.from_env()
    if args.layers or args.tiny:
        return run_generation(cfg, args, build_model(cfg, args, tp, arch), tp)
    model = registry.load_model(args.model, tp, tp.device, getattr(torch, args.dtype), args.moe_parallel,
                                weights_folder=args.checkpoint)
    return run_generation(cfg, args, model, tp)


if __name__ == "__main__":
    sys.exit(main())
