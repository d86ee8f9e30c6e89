"""Command line.

    python -m runnburn_b200 generate --model PATH --prompt 1,2,3 [-n 16] [--dtype bfloat16] [--max-ctx N]

PATH: a .gguf file or a folder with config.json and model.safetensors.  Token ids in, greedy token ids out.
"""
from __future__ import annotations

import argparse
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m runnburn_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="greedy continuation of a prompt of token ids")
    g.add_argument("--model", required=True)
    g.add_argument("--prompt", required=True, help="token ids with commas between them")
    g.add_argument("-n", type=int, default=16, help="tokens to generate")
    g.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    g.add_argument("--max-ctx", type=int, default=0)
    a = ap.parse_args(argv)
    from .registry import load_model
    prompt = [int(t) for t in a.prompt.split(",")]
    dec = load_model(a.model, a.max_ctx, a.dtype)
    print(",".join(str(t) for t in dec.generate(prompt, a.n)))
    dec.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
