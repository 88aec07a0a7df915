"""Trace replay: given token ids go through a model step by step, logits come out; nothing is sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

One JSON object a line on standard input:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
An entry brings a request's next tokens and the places among them whose logits are wanted; `end` lists the requests
that are finished after the step. A step with something wanted writes <out>/<step>.f32 (little-endian fp32, wanted x
vocab, in the order of the entries); every step prints "done <step>". The model, its step function, its caches and its
kernels are those of generation (dejavu_b200.generation.SequencePool).
Exit codes: 0 at the end of the input, 3 if the model does not run in the dtype that is asked for.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids through a model.")
    ap.add_argument("--model", required=True, help="folder with config.json and .safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens the live requests hold at any time")
    args = ap.parse_args(argv)

    import torch

    from . import build, registry
    from .generation import SequencePool

    entry = registry.entry_for(registry.read_config(args.model))
    dtype = getattr(torch, args.dtype)
    if dtype not in entry.dtypes:
        print(f"this model does not run in {args.dtype}", file=sys.stderr)
        return 3
    build.build(libs=(entry.library,))  # a fresh checkout has no kernels yet
    device = torch.device("cuda", 0)
    pool = SequencePool(registry.load_model(args.model, dtype, device), args.max_tokens, device)
    for line in sys.stdin:
        if not line.strip():
            continue
        work = json.loads(line)
        parts = []
        for e in work["entries"]:
            logits = pool.run(e["id"], e["tokens"], e["want"])
            if e["want"]:
                parts.append(logits)
        if parts:
            data = torch.cat(parts).float().cpu().contiguous().numpy().astype("<f4")
            path = os.path.join(args.out, f"{work['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(data.tobytes())
            os.replace(path + ".part", path)
        else:
            torch.cuda.synchronize()
        for request in work["end"]:
            pool.end(request)
        print(f"done {work['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
