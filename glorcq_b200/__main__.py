"""Command line:

    python -m glorcq_b200 generate --model DIR --tokens 5,17,3 --max-new-tokens 32
    python -m glorcq_b200 trace --model DIR --dtype bfloat16 --out DIR --max-tokens N < steps.jsonl
"""

from __future__ import annotations

import argparse
import sys


def generate(args):
    import torch
    from .graph_wrapper import GLoRCQGraphWrapper
    from .registry import load_model
    model = load_model(args.model, "cuda:0", args.dtype)
    prompt = [int(t) for t in args.tokens.split(",")]
    w = GLoRCQGraphWrapper(model, max_batch_size=1, max_seq_len=max(16, len(prompt) + args.max_new_tokens))
    ids, _ = w.generate(torch.tensor([prompt], device=w.device), max_new_tokens=args.max_new_tokens)
    print(",".join(str(t) for t in ids[0, len(prompt):].tolist()))
    if args.timing:
        print(f"prompt {len(prompt)} tokens: {w.last_prefill_seconds * 1e3:.2f} ms; decode: "
              f"{(args.max_new_tokens - 1) / max(w.last_decode_seconds, 1e-9):.1f} tokens/s", file=sys.stderr)
    return 0


def trace(args):
    from .trace import main as run
    return run(args)


def main(argv=None):
    ap = argparse.ArgumentParser(prog="glorcq_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy generation from token ids")
    g.add_argument("--model", required=True, help="checkpoint folder")
    g.add_argument("--tokens", required=True, help="prompt token ids, comma separated")
    g.add_argument("--max-new-tokens", type=int, default=32)
    g.add_argument("--dtype", choices=["bfloat16", "float16", "float32"], default=None, help="default: the design's own")
    g.add_argument("--timing", action="store_true", help="print prompt and decode times to standard error")
    t = sub.add_parser("trace", help="replay given tokens step by step (steps on standard input) and write logits")
    t.add_argument("--model", required=True, help="checkpoint folder")
    t.add_argument("--dtype", choices=["bfloat16", "float16", "float32"], default=None)
    t.add_argument("--out", required=True, help="folder for <step>.f32")
    t.add_argument("--max-tokens", type=int, default=4096, help="most tokens a live request holds")
    args = ap.parse_args(argv)
    return {"generate": generate, "trace": trace}[args.command](args)


if __name__ == "__main__":
    sys.exit(main())
