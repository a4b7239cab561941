"""Greedy generation from the command line, for every model the registry opens (token ids in, token ids out).

    python -m juno_b200.generate MODEL --ids 1,17,5 [--ids 9,2] --steps 32 [--dtype default|f32] [--token-by-token]

MODEL is a folder (config.json + model.safetensors) or a GGUF file.  Several --ids run as one decode batch; one line of ids per
prompt is printed.
"""
from __future__ import annotations

import argparse
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="juno_b200.generate", description="greedy continuation of prompts of token ids")
    ap.add_argument("model")
    ap.add_argument("--ids", action="append", required=True, help="comma-separated token ids of one prompt")
    ap.add_argument("--steps", type=int, default=16)
    ap.add_argument("--dtype", choices=["default", "f32"], default="default")
    ap.add_argument("--token-by-token", action="store_true", help="feed the prompts through decode steps instead of the prompt path")
    a = ap.parse_args(argv)
    from .handler import B200InferencePipeline, B200TransformerHandler, generate_greedy
    prompts = [[int(t) for t in s.split(",")] for s in a.ids]
    room = max(len(p) for p in prompts) + a.steps + 1
    h = B200TransformerHandler.open(a.model, max_batch=max(2, len(prompts)), max_seqs=len(prompts), max_ctx=room, dtype=a.dtype)
    names = [str(i) for i in range(len(prompts))]
    if len(prompts) == 1:
        out = [generate_greedy(B200InferencePipeline(h), "0", prompts[0], a.steps, chunked_prefill=not a.token_by_token)]
    else:
        for n, p in zip(names, prompts):
            if len(p) > 1 and not a.token_by_token:
                h.prefill(n, p[:-1], 0)
            else:
                for i, t in enumerate(p[:-1]):
                    h.forward_batch([n], [[t]], [i], want_logits=False, want_argmax=True)
        out = h.decode_greedy(names, [p[-1] for p in prompts], [len(p) - 1 for p in prompts], a.steps).T.tolist()
    for ids in out:
        print(",".join(map(str, ids)))
    h.release_gpu_resources()
    return 0


if __name__ == "__main__":
    sys.exit(main())
