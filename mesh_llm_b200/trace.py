"""Replays a trace of token ids through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps

Steps come on standard input, one JSON object a line:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
Every entry's tokens run from where the request stands; the logits at the wanted places go to <out>/<step>.f32
(little-endian 32-bit floats, in the order of the entries and of "want").  "done <step>" is printed after each step.
Exit code 3: the model does not run in 32-bit.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

SLOTS = 8


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="checkpoint folder (config.json, model.safetensors) or GGUF file")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens live requests hold at any time")
    ap.add_argument("--ubatch", type=int, default=512, help="tokens per forward pass")
    args = ap.parse_args(argv)

    from .engine import Engine, PrecisionError, open_stage

    n_ctx = max(1, args.max_tokens)
    try:
        stage = open_stage(args.model, args.dtype, n_ctx=n_ctx, n_seq=SLOTS, n_ubatch=max(1, min(args.ubatch, n_ctx)))
    except PrecisionError as e:
        print(e, file=sys.stderr)
        return 3
    eng = Engine(stage)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = [eng.feed(e["id"], e["tokens"], e["want"]) for e in step["entries"]]
        if rows and sum(len(r) for r in rows):
            eng.check()
            with open(os.path.join(args.out, "%d.f32" % step["step"]), "wb") as f:
                f.write(np.concatenate(rows).astype("<f4").tobytes())
        for rid in step["end"]:
            if rid in eng.live:
                eng.end(rid)
        print("done %d" % step["step"], flush=True)
    stage.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
