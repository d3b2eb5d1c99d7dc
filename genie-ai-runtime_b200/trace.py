"""Replays a token trace through a model and writes logits: `bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR
--max-tokens N`.

Standard input is JSON lines, {"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [...]}: an entry
appends tokens to a request and lists the indices into them that need logits; `end` names requests to release.  Logits go to
<out>/<n>.f32 (float32 rows, entry by entry, index by index), no file for a step that needs none; `done n` is printed after
each step.  Exit code 3: the model does not run in the requested number format.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

from .engine import Engine
from .registry import DtypeError, check_config, read_config


def replay(engine, lines, out_dir, report=print):
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = [engine.feed(e["id"], e["tokens"], e["want"]) for e in step["entries"] if e["tokens"]]
        rows = [r for r in rows if len(r)]
        if rows:
            np.concatenate(rows).astype("<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        for request in step.get("end", ()):
            engine.end(request)
        report(f"done {step['step']}")


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a token trace (JSON lines on standard input) and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, help="number format, e.g. bfloat16 or float32")
    ap.add_argument("--out", required=True, help="folder for the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="cache size: positions a request may fill")
    a = ap.parse_args(argv)
    try:
        check_config(read_config(a.model), a.dtype)
    except DtypeError as e:
        print(e, file=sys.stderr)
        return 3
    engine = Engine(a.model, a.dtype, max_context=max(a.max_tokens, 1))
    replay(engine, sys.stdin, a.out, lambda text: print(text, flush=True))
    engine.close()
    return 0
