"""Trace replay: feeds given token ids through a model step by step and writes logits.  Nothing is sampled; the steps
run on ``StackEngine``, the engine that generation uses.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps

Standard input holds one JSON object per line,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

the next tokens of each sequence, the places among them whose logits are wanted, and the sequences that are finished
after the step.  Wanted logits go to OUT/<step>.f32 (little-endian fp32 [wanted, vocab], in the order of entries and
places); ``done <step>`` is printed after every step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

from ..models.registry import load_folder
from .stack import StackEngine

MAX_LIVE = 64                # sequences that can be open at once


def replay(engine: StackEngine, lines, out_dir: str, emit) -> None:
    """Runs the steps in ``lines``; ``emit(step)`` is called after each."""
    slots: dict[str, int] = {}
    for line in lines:
        if not line.strip():
            continue
        msg = json.loads(line)
        entries = []
        for e in msg["entries"]:
            if e["id"] not in slots:
                slots[e["id"]] = engine.open()
            entries.append((slots[e["id"]], e["tokens"], e["want"]))
        logits = engine.step(entries)
        if logits.shape[0]:
            path = os.path.join(out_dir, f"{msg['step']}.f32")
            with open(path, "wb") as f:
                f.write(logits.float().cpu().contiguous().numpy().astype("<f4").tobytes())
        elif engine.device.type == "cuda":
            torch.cuda.synchronize()
        for name in msg.get("end", []):
            if name in slots:
                engine.close(slots.pop(name))
        emit(msg["step"])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=8192, help="most tokens that live sequences hold at any time")
    ap.add_argument("--page-size", type=int, default=64)
    args = ap.parse_args(argv)
    if not torch.cuda.is_available():
        print("trace_run: needs a CUDA device", file=sys.stderr)
        return 2
    dtype = getattr(torch, args.dtype)
    model = load_folder(args.model, torch.device("cuda", torch.cuda.current_device()), dtype)
    engine = StackEngine(model, MAX_LIVE, max(args.max_tokens, 1), args.page_size, pool_tokens=max(args.max_tokens, 1))

    def emit(step):
        print(f"done {step}", flush=True)
    replay(engine, sys.stdin, args.out, emit)
    return 0
