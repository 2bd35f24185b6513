"""Trace replay: steps of given token ids in, wanted logits out, through the same Engine that serves
generation (bin/trace_run is the command)."""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

from .engine import Engine
from .registry import load_model

MAX_ROWS = 1024              # tokens of one session step; longer prompts run in portions


def replay(engine: Engine, lines, out_dir: str, report) -> None:
    live = None                                            # the request the session's state belongs to
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = step["entries"]
        if len(entries) > 1:
            raise ValueError("a step holds one request: the session keeps the state of one sequence")
        rows = []
        for entry in entries:
            if live is not None and entry["id"] != live:
                raise ValueError(f"request {entry['id']!r} starts before {live!r} has ended")
            live = entry["id"]
            rows.append(engine.feed(entry["tokens"], entry["want"]))
        if rows and rows[0].shape[0]:
            np.concatenate(rows).astype("<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        if live is not None and live in step.get("end", ()):
            engine.end()
            live = None
        report(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids through a model.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens a request holds at any time")
    args = ap.parse_args(argv)
    limit = max(args.max_tokens, 1)
    model = load_model(args.model, dtype=args.dtype, max_rows=min(MAX_ROWS, limit), max_tokens=limit)

    def report(text):
        print(text, flush=True)
    replay(Engine(model, greedy=False), sys.stdin, args.out, report)
    return 0
