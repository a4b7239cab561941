"""Replays a trace of token ids through a model: the command behind bin/trace_run.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come as JSON lines on standard input,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

each entry a request's next tokens and the places among them whose logits are wanted.  A step with wanted places leaves
OUT/<step>.f32 (little-endian FP32 [wanted, vocab]); every step is answered with a line "done <step>".  Requests named in
"end" give their pages and slot back.  Everything runs through the handler that generation uses: a single token is a decode
step, more tokens a portion of a prompt.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


def run(handler, lines, out_dir: str, answer) -> None:
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for e in step["entries"]:
            if not e["tokens"]:
                continue
            logits = handler.feed(e["id"], e["tokens"], e.get("want", ()))
            if len(logits):
                rows.append(logits)
        if rows:
            np.concatenate(rows).astype("<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        for rid in step.get("end", ()):
            handler.evict(rid)
        answer(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids through a model, step by step")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=4, help="most requests that are live at any time")
    a = ap.parse_args(argv)
    from . import build
    build.build()
    from .handler import B200TransformerHandler
    h = B200TransformerHandler.open(a.model, max_batch=1, max_seqs=a.max_requests, max_ctx=max(16, a.max_tokens),
                                    dtype="f32" if a.dtype == "float32" else "default")

    def answer(text: str) -> None:
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    run(h, sys.stdin, a.out, answer)
    h.release_gpu_resources()
    return 0


if __name__ == "__main__":
    sys.exit(main())
