"""Trace runner: replays given token streams through a model, step by step, and writes logits.

  trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N [--device cuda[:I]|cpu] [--page-size P]

Steps come from standard input, one JSON object a line:

  {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step are one batch.  For a step that wants logits the runner writes OUT/<step>.f32 (little-endian fp32
rows [wanted, vocab], in the order of the entries and of `want`); after every step it prints `done <step>`.  The
model, its caches and its kernels are those of the serving engine: the page pool holds N tokens, there are four sequence
slots, and the requests named in `end` give theirs back after the step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import List, Optional

SLOTS = 4


def build_replay(model_dir: str, dtype: str, max_tokens: int, device: str, page_size: int):
    import torch

    from ..models.registry import RunnerLimits, architecture_of
    from ..runtime.engine import EngineConfig
    from ..runtime.replay import ReplayEngine
    from ..runtime.scheduler import SchedulerConfig
    arch = architecture_of(model_dir)
    dt = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype]
    if device.startswith("cuda"):
        if not torch.cuda.is_available():
            raise SystemExit("trace_run: no CUDA device")
        torch.backends.cuda.matmul.allow_tf32 = False
        if dt not in arch.dtypes:
            print(f"trace_run: {arch.name} does not run in {dtype}", file=sys.stderr)
            raise SystemExit(3)
        device = device if ":" in device else "cuda:0"
        torch.cuda.set_device(torch.device(device))
        from ..ops import _lib
        _lib.use_component(arch.component)
    weights = arch.load(model_dir, device, dt)
    pages = (max_tokens + page_size - 1) // page_size
    ctx = (pages + 1) * page_size
    rows = pages * page_size
    runner = arch.runner(weights, RunnerLimits(pages, page_size, rows, SLOTS, ctx), device=device,
                         full_logit_rows=min(256, rows))
    sched = SchedulerConfig(max_active_sequences=SLOTS, max_decode_batch=min(SLOTS, rows), max_batch_tokens=rows,
                            prefill_chunk_size=rows, ctx_size=ctx)
    return ReplayEngine(runner, EngineConfig(scheduler=sched, kv_pages=pages, page_size=page_size))


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay token streams through a model and write logits")
    ap.add_argument("--model", required=True, help="checkpoint directory (config.json and safetensors)")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="directory for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="most tokens live requests hold at any time (each rounded up to whole pages)")
    ap.add_argument("--device", default="cuda")
    ap.add_argument("--page-size", type=int, default=64)
    args = ap.parse_args(argv)
    if args.max_tokens <= 0 or args.page_size <= 0:
        ap.error("--max-tokens and --page-size must be positive")
    import numpy as np

    from ..io.safetensors import CheckpointError
    from ..runtime.replay import ReplayEntry
    try:
        engine = build_replay(args.model, args.dtype, args.max_tokens, args.device, args.page_size)
    except CheckpointError as exc:
        print(f"error: {exc}", file=sys.stderr)
        return 2
    cuda = args.device.startswith("cuda")
    if cuda:
        from ..ops._lib import raise_on_status
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [ReplayEntry(str(e["id"]), [int(t) for t in e["tokens"]], [int(w) for w in e.get("want", ())])
                   for e in step.get("entries", ())]
        rows = engine.replay(entries, [str(i) for i in step.get("end", ())])
        if cuda:
            raise_on_status()
        if any(e.want for e in entries):
            path = os.path.join(args.out, f"{step['step']}.f32")
            np.concatenate(rows).astype("<f4").tofile(path)
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
