"""Greedy generation from token ids, with a checkpoint folder or a GGUF file:

    python -m mesh_llm_b200.generate --model PATH --tokens 5,17,3 [--tokens 9,2] -n 32

One line of comma-separated new ids per prompt.
"""
from __future__ import annotations

import argparse
import sys


def main(argv=None):
    ap = argparse.ArgumentParser(prog="python -m mesh_llm_b200.generate", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="checkpoint folder (config.json, model.safetensors) or GGUF file")
    ap.add_argument("--tokens", action="append", required=True, help="a prompt: token ids with commas between them; repeatable")
    ap.add_argument("-n", "--max-new", type=int, default=32)
    ap.add_argument("--stop", default="", help="token ids that end a sequence")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--n-ctx", type=int, default=0, help="room per sequence (default: the longest prompt + max-new)")
    ap.add_argument("--slots", type=int, default=8, help="sequences in flight")
    ap.add_argument("--ubatch", type=int, default=512, help="tokens per forward pass of a prompt")
    args = ap.parse_args(argv)

    from .engine import Engine, open_stage

    ids = lambda s: [int(t) for t in s.split(",") if t.strip()]  # noqa: E731
    prompts = [ids(t) for t in args.tokens]
    n_ctx = args.n_ctx or max(len(p) for p in prompts) + args.max_new
    n_seq = max(1, min(args.slots, len(prompts)))
    stage = open_stage(args.model, args.dtype, n_ctx=n_ctx, n_seq=n_seq, n_ubatch=max(n_seq, min(args.ubatch, n_ctx)))
    for new in Engine(stage).generate(prompts, args.max_new, ids(args.stop)):
        print(",".join(str(t) for t in new))
    return 0


if __name__ == "__main__":
    sys.exit(main())
