"""Greedy generation from the command line, for any model of the registry.

    python -m fastkernels_b200.generate --model DIR --prompt 5,17,3 [--prompt ...]
        [--max-new-tokens N] [--dtype bfloat16|float32] [--chunk-tokens C]

Prompts are token ids (there is no tokenizer here); one line of new token ids is printed
per prompt.  Runs DecodeEngine.prefill and CUDA-graph decode steps.
"""
from __future__ import annotations

import argparse
import sys

import torch

from .engine import DecodeEngine


def parse_args(argv=None):
    ap = argparse.ArgumentParser(prog="generate", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors")
    ap.add_argument("--prompt", action="append", required=True,
                    help="token ids with commas between; repeat for a batch")
    ap.add_argument("--max-new-tokens", type=int, default=16)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--chunk-tokens", type=int, default=None,
                    help="most prompt tokens per forward")
    return ap.parse_args(argv)


def main(argv=None, stdout=None) -> int:
    args = parse_args(argv)
    prompts = [[int(t) for t in p.split(",")] for p in args.prompt]
    longest = max(len(p) for p in prompts) + args.max_new_tokens
    eng = DecodeEngine.from_folder(args.model, dtype=getattr(torch, args.dtype),
                                   max_tokens=longest * len(prompts), max_num_seqs=len(prompts))
    if args.max_new_tokens > 0:
        eng.prefill(prompts, chunk_tokens=args.chunk_tokens)
    if args.max_new_tokens > 1:
        eng.capture_cudagraph([len(prompts)])
        eng.decode(args.max_new_tokens - 1)
    for s in eng.seqs:
        print(",".join(str(t) for t in s.output), file=stdout or sys.stdout)
    return 0


if __name__ == "__main__":
    sys.exit(main())
