"""Replay a trace of token portions through a model and write the logits it asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every entry feeds the next tokens of its sequence through the model's step function (nfai_forward) from the cache and the
state earlier steps left; `want` are the places among them whose logits go into DIR/<step>.f32 ([wanted][vocabulary],
little-endian float32, in the order of the entries). `end` lists the sequences that are finished. After every step the line
"done <step>" is printed. One sequence occupies the model; when another one is continued in between, the first is kept as
a snapshot and brought back when its turn comes.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Optional

import numpy as np


class Sequences:
    """Several sequences on one model: the active one lives in its cache, the others as snapshots."""

    def __init__(self, model):
        self.model = model
        self.active: Optional[str] = None
        self.parked: Dict[str, object] = {}

    def select(self, name: str):
        if name == self.active:
            return
        if self.active is not None:
            self.parked[self.active] = self.model.snapshot()
        snap = self.parked.pop(name, None)
        if snap is None:
            self.model.reset()
        else:
            snap.restore()
            snap.close()
        self.active = name

    def end(self, name: str):
        if name == self.active:
            self.active = None
        snap = self.parked.pop(name, None)
        if snap is not None:
            snap.close()


def replay(model, lines, out_dir: str, report) -> None:
    seqs = Sequences(model)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        rows: List[np.ndarray] = []
        for entry in step["entries"]:
            seqs.select(entry["id"])
            want = [int(w) for w in entry.get("want", [])]
            if not entry["tokens"]:
                continue
            order = sorted(set(want))
            got = model.forward(entry["tokens"], order)
            rows += [got[order.index(w)] for w in want]
        for name in step.get("end", []):
            seqs.end(name)
        if rows:
            part = os.path.join(out_dir, f"{step['step']}.f32.part")
            np.stack(rows).astype("<f4").tofile(part)
            os.replace(part, os.path.join(out_dir, f"{step['step']}.f32"))
        report(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token portions through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=4096, help="capacity of the cache in tokens")
    ap.add_argument("--device", type=int, default=0)
    args = ap.parse_args(argv)

    from . import build
    build.build()  # compiles what is missing or out of date; nothing otherwise
    from .api import CudaContext, ModelOptions
    from .registry import architecture_of, try_create

    ctx = CudaContext(args.device)
    model = try_create(ctx, ModelOptions(ModelPath=args.model, KVCacheSize=max(1, args.max_tokens),
                                         WeightDType="bf16" if args.dtype == "bfloat16" else "f32"))
    if model is None:
        print(f"no model class for architecture {architecture_of(args.model)!r}", file=sys.stderr)
        return 2
    os.makedirs(args.out, exist_ok=True)
    replay(model, sys.stdin, args.out, lambda text: print(text, flush=True))
    model.Dispose()
    ctx.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
