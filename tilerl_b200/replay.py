"""Replay of a recorded trace: given token ids go through the engine step by step, logits come out.

``python -m tilerl_b200.replay --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N`` (``bin/trace_run``)
reads steps from standard input, one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

runs each as one tick (:meth:`Engine.feed`: the scheduler's pools, captured decode ticks and model forward),
writes the wanted logits to ``OUT/<step>.f32`` (little-endian fp32 ``[wanted, vocab]``) and prints
``done <step>``.  Nothing is sampled.  No counterpart in the reference.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Iterable, Optional, TextIO

import torch

from .config import get_config
from .engine import Engine
from .factory import build_engine, build_model, make_ops
from .ops.ref import KV_BLOCK

SLOTS = 4                  # live requests
EXIT_NO_DTYPE = 3


def open_engine(model_dir: str, dtype: torch.dtype, max_tokens: int, device: str, slots: int = SLOTS) -> Engine:
    """An engine whose KV pool holds ``max_tokens`` tokens (plus the pad page) and ``slots`` live requests."""
    cfg = get_config(model_dir)
    ops = make_ops(device)
    model = build_model(cfg, device, checkpoint=model_dir, dtype=dtype, ops=ops if device != "cpu" else None)
    pages = (max_tokens + KV_BLOCK - 1) // KV_BLOCK
    return build_engine(model, ops, device=device, blocks=pages + 1, slots=slots, max_ctx=max(1, pages) * KV_BLOCK, prefix=False)


def replay(eng: Engine, lines: Iterable[str], out_dir: str, answers: TextIO) -> int:
    """Run every step of ``lines``; returns how many there were."""
    n = 0
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = eng.feed([(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]], step.get("end", []))
        if logits is not None:
            path = os.path.join(out_dir, f"{step['step']}.f32")
            logits.detach().float().cpu().contiguous().numpy().astype("<f4").tofile(path)
        print(f"done {step['step']}", file=answers, flush=True)
        n += 1
    return n


def main(argv: Optional[list] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay given tokens through the engine, write logits")
    ap.add_argument("--model", required=True, help="directory with config.json and safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory of the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default=None, help="cuda | cpu (default: cuda; cpu runs the reference backend)")
    args = ap.parse_args(argv)
    device = args.device or "cuda"
    if device != "cpu":
        from . import build
        from .ops import native
        native.use(build.ensure(getattr(get_config(args.model), "architecture", "")))
    try:
        eng = open_engine(args.model, getattr(torch, args.dtype), args.max_tokens, device)
    except ValueError as e:
        if "does not run in" in str(e):
            print(str(e), file=sys.stderr)
            return EXIT_NO_DTYPE
        raise
    os.makedirs(args.out, exist_ok=True)
    replay(eng, sys.stdin, args.out, sys.stdout)
    return 0


if __name__ == "__main__":
    sys.exit(main())
