"""Greedy generation from the command line.

    python genie-ai-runtime_b200/generate.py --model DIR [--dtype bfloat16] [--new 32] PROMPT [PROMPT ...]

DIR holds config.json and model.safetensors of a registered architecture; a prompt is comma-separated token ids (there is no
tokenizer here).  Prints one JSON line per prompt."""
import argparse
import json
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)


def main(argv=None):
    from __graft_entry__ import load_package
    ap = argparse.ArgumentParser(description="Greedy generation from token-id prompts.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", help="number format (default: the architecture's first)")
    ap.add_argument("--new", type=int, default=32, help="tokens to generate per prompt")
    ap.add_argument("--max-context", type=int, help="positions a request may hold (default: what the prompts need)")
    ap.add_argument("prompts", nargs="+", metavar="PROMPT", help="comma-separated token ids")
    a = ap.parse_args(argv)
    prompts = [[int(t) for t in p.split(",")] for p in a.prompts]
    jb = load_package()
    engine = jb.engine.Engine(a.model, a.dtype, a.max_context or max(len(p) for p in prompts) + a.new)
    for p, out in zip(prompts, engine.generate(prompts, a.new)):
        print(json.dumps({"prompt": p, "tokens": out}))
    engine.close()


if __name__ == "__main__":
    main()
