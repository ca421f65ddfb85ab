"""Replays a trace: given token ids go through a model step by step, logits come out.  Nothing is sampled.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  <  steps.jsonl

A step is one JSON line {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}: every entry's tokens continue its
sequence, "want" lists the places among them whose logits are written (OUT/<n>.f32, little-endian fp32, entries in order),
"end" the sequences that are given back afterwards.  "done <n>" follows on standard output."""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

MAX_LIVE = 16          # sequences at a time
MAX_STEP_TOKENS = 2048  # longer steps run in passes of this many tokens


def replay(model, lines, out_dir, emit):
    row_of, ids = {}, []  # id -> batch row; ids[row] = id
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries, want, base = [], [], 0
        for e in step["entries"]:
            if e["id"] not in row_of:
                row_of[e["id"]] = model.open()
                ids.append(e["id"])
            if not e["tokens"]:
                continue
            entries.append((row_of[e["id"]], e["tokens"]))
            want += [base + w for w in e["want"]]
            base += len(e["tokens"])
        if entries:
            _, logits = model.step(entries, want)
            if want:
                logits.astype("<f4", copy=False).tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        for i in step.get("end", []):
            if i not in row_of:
                continue
            row = row_of.pop(i)
            moved = model.retire(row)
            last = ids.pop()
            if moved >= 0:
                ids[row] = last
                row_of[last] = row
        emit(f"done {step['step']}")


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay given tokens through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens that live sequences hold at any time")
    a = ap.parse_args(argv)
    from .registry import load_model
    n = max(a.max_tokens, 1)
    model = load_model(a.model, a.dtype, max_batch=MAX_LIVE, max_context=n, max_step_tokens=min(MAX_STEP_TOKENS, max(n, MAX_LIVE)),
                       pool_pages=-(-n // 64) + MAX_LIVE)

    def emit(line):
        print(line, flush=True)

    replay(model, sys.stdin, a.out, emit)
    model.close()
    return 0
