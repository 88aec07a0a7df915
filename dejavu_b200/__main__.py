"""Command line:

    python -m dejavu_b200 generate --model DIR --tokens 5,17,3 --max-new-tokens 32 [--dtype bfloat16] [--cuda-graph]
                                   [--prompt-chunk N]
    python -m dejavu_b200 trace --model DIR --dtype bfloat16 --out DIR --max-tokens N < steps.jsonl

`generate` prints the new token ids of a greedy continuation, one line per prompt; several prompts of one length
(separated by ';') run as a batch.
"""
from __future__ import annotations

import argparse
import sys


def generate(argv) -> int:
    ap = argparse.ArgumentParser(prog="python -m dejavu_b200 generate", description="Greedy generation from token ids.")
    ap.add_argument("--model", required=True, help="folder with config.json and .safetensors")
    ap.add_argument("--tokens", required=True, help="prompt ids, comma separated; prompts of one length separated by ';'")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--dtype", default=None, choices=["bfloat16", "float16", "float32"])
    ap.add_argument("--cuda-graph", action="store_true", help="decode through one captured CUDA graph")
    ap.add_argument("--prompt-chunk", type=int, default=None, help="run the prompt in portions of at most this many tokens")
    args = ap.parse_args(argv)

    import torch

    from . import registry

    model = registry.load_model(args.model, None if args.dtype is None else getattr(torch, args.dtype))
    prompts = [[int(t) for t in p.split(",")] for p in args.tokens.split(";")]
    if len({len(p) for p in prompts}) != 1:
        ap.error("the prompts of a batch have one length")
    vocab = model.config.vocab_size
    if any(not 0 <= t < vocab for p in prompts for t in p):
        ap.error(f"token ids are 0 .. {vocab - 1}")
    ids = torch.tensor(prompts, dtype=torch.long, device="cuda")
    out = model.generate(ids, ids.size(1) + args.max_new_tokens, cg=args.cuda_graph, vocab_size=vocab,
                         prompt_chunk=args.prompt_chunk)
    for row in out[:, ids.size(1):].tolist():
        print(",".join(map(str, row)))
    return 0


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else argv
    if argv and argv[0] == "generate":
        return generate(argv[1:])
    if argv and argv[0] == "trace":
        from .trace import main as trace

        return trace(argv[1:])
    print(__doc__)
    return 2


if __name__ == "__main__":
    sys.exit(main())
