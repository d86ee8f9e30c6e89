"""Replays a trace: token ids are fed to a model step by step and logits are written.

    python -m runnburn_b200.trace --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come on standard input, one JSON object a line:
    {"step": 4, "entries": [{"id": "q7", "tokens": [12, 9], "want": [1]}], "end": ["q7"]}
`want` are places among the step's tokens; a request named in `end` is over after the step.
For a step that wants logits, OUT/<step>.f32 receives them ([wanted, vocab], little-endian f32); after
every step 'done <step>' is printed.  One sequence is live at a time: a request runs until it ends.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from pathlib import Path


def replay(dec, lines, out_dir: Path, echo) -> None:
    import numpy as np
    live, pos = None, 0
    for line in lines:
        if not line.strip():
            continue
        st = json.loads(line)
        rows = []
        for e in st["entries"]:
            tokens, want = e["tokens"], e.get("want", [])
            if e["id"] != live:
                if live is not None:
                    raise ValueError(f"request {e['id']!r} starts before {live!r} has ended")
                live, pos = e["id"], 0
                dec.reset()
            if len(tokens) == 1 and pos > 0:
                _, logits = dec.step(tokens[0], pos, want_logits=True)
                rows += [logits] * len(want)
            elif tokens:
                logits, _ = dec.prefill_logits(tokens, pos, want)
                rows += list(logits)
            pos += len(tokens)
        if rows:
            part = out_dir / f".{st['step']}.part"
            np.stack(rows).astype("<f4").tofile(part)
            os.replace(part, out_dir / f"{st['step']}.f32")
        if live in st.get("end", []):
            live, pos = None, 0
            dec.reset()
        echo(f"done {st['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids and write logits.")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=4096)
    a = ap.parse_args(argv)
    from .build import build_library
    build_library()
    from .registry import load_model
    dec = load_model(a.model, max_ctx=max(a.max_tokens, 1), dtype=a.dtype)
    replay(dec, sys.stdin, Path(a.out), lambda text: print(text, flush=True))
    dec.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
