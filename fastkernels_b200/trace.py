"""Replay a trace: given token ids through a model, step by step, logits to files.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps

One JSON object per input line, {"step": n, "entries": [{"id", "tokens", "want"}],
"end": [ids]}: the next tokens of each request, the places among them whose logits
are wanted, and the requests that are finished.  Wanted logits go to DIR/<n>.f32
(little-endian fp32, in the order of the entries), and 'done <n>' to standard output.
Nothing is sampled; the tokens run through DecodeEngine.feed.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

from .engine import DecodeEngine

MAX_SEQS = 64


def parse_args(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=8192,
                    help="most tokens that live requests hold at any time")
    return ap.parse_args(argv)


def make_engine(folder, dtype, max_tokens) -> DecodeEngine:
    eng = DecodeEngine.from_folder(folder, dtype=dtype, max_tokens=max_tokens,
                                   max_num_seqs=MAX_SEQS)
    eng.capture_cudagraph([1])
    return eng


def main(argv=None, stdin=None, stdout=None) -> int:
    args = parse_args(argv)
    stdin, stdout = stdin or sys.stdin, stdout or sys.stdout
    dtype = getattr(torch, args.dtype)
    eng = make_engine(args.model, dtype, args.max_tokens)
    live = {}
    for line in stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = eng.open_sequence()
            entries.append((live[e["id"]], e["tokens"]))
        logits = eng.feed(entries, [e["want"] for e in step["entries"]]) if entries else []
        rows = [x for x in logits if x.shape[0]]
        if rows:
            data = torch.cat(rows).contiguous().numpy().astype("<f4").tobytes()
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as f:
                f.write(data)
        for name in step.get("end", []):
            eng.finish(live.pop(name))
        status = eng.device_status()
        if status:
            raise RuntimeError(f"device status word {status} (fk_device_status bits)")
        print(f"done {step['step']}", file=stdout, flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
