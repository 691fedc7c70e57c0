"""Replay of recorded steps through the serving engine (command line: bin/trace_run).

The engine is the one that generates: `GenerationEngine.run_step` takes each step's entries as one batch, decode steps
replay the captured graph, and the cache pool holds `max_tokens` tokens and four sequences, so blocks and state slots
are reused as requests end.
"""

from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, Iterable, List, Optional, TextIO

import torch

from .engine import GenerationEngine, StepEntry
from .kv_cache import BLOCK_SIZE, SequenceState

MAX_REQUESTS = 4


class TraceReplay:
    def __init__(self, engine: GenerationEngine):
        self.engine = engine
        self.live: Dict[str, SequenceState] = {}

    def step(self, spec: dict) -> Optional[torch.Tensor]:
        """Run one step; returns the wanted logits (fp32 [wanted, vocab], CPU) or None."""
        entries: List[StepEntry] = []
        for e in spec["entries"]:
            if e["id"] not in self.live:
                self.live[e["id"]] = self.engine.open_request()
            entries.append(StepEntry(self.live[e["id"]], e["tokens"], e.get("want") or ()))
        logits = self.engine.run_step(entries)
        out = None if logits is None else logits.float().cpu()
        ended = [self.live.pop(i) for i in spec.get("end") or () if i in self.live]
        if ended:
            self.engine.release(ended)
        return out


def replay(engine: GenerationEngine, lines: Iterable[str], out_dir: str, log: TextIO) -> None:
    run = TraceReplay(engine)
    for line in lines:
        if not line.strip():
            continue
        spec = json.loads(line)
        logits = run.step(spec)
        if logits is not None:
            path = os.path.join(out_dir, f"{spec['step']}.f32")
            with open(path, "wb") as f:
                f.write(logits.contiguous().numpy().astype("<f4").tobytes())
        print(f"done {spec['step']}", file=log, flush=True)


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(description="replay steps of token ids (JSON lines on standard input) and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default="cuda", help="cpu: the operators' PyTorch statements (development)")
    args = ap.parse_args(argv)
    from ..ops import KernelLibraryError, _lib, raise_on_device_error
    from . import registry

    on_gpu = torch.device(args.device).type == "cuda"
    if on_gpu:
        if not torch.cuda.is_available():
            print("no CUDA device", file=sys.stderr)
            return 1
        _lib.use_serving_subset()
    try:
        model = registry.load_model(args.model, device=args.device, dtype=getattr(torch, args.dtype))
    except KernelLibraryError as e:
        print(e, file=sys.stderr)
        return 1
    tokens = (args.max_tokens + BLOCK_SIZE - 1) // BLOCK_SIZE * BLOCK_SIZE
    engine = GenerationEngine(model, max_batch=MAX_REQUESTS, max_seq_len=tokens, num_blocks=tokens // BLOCK_SIZE)
    replay(engine, sys.stdin, args.out, sys.stdout)
    if on_gpu:
        raise_on_device_error()
    return 0
