"""Command line: `python -m loom_b200 generate --model DIR --tokens 1,2,3 [--tokens ...] --max-new 16`, `python -m loom_b200 models`,
`python -m loom_b200 trace ...` (the same as bin/trace_run)."""
from __future__ import annotations

import argparse
import json
import sys


def generate(args) -> int:
    from . import Context, models

    prompts = [[int(t) for t in p.split(",")] for p in args.tokens]
    ctx = Context(args.device)
    dec = models.load(ctx, args.model, args.dtype, args.max_seq_len, batch=len(prompts))
    if len(prompts) == 1:
        tokens, m = dec.generate(prompts[0], args.max_new)
        print(json.dumps({"tokens": tokens.tolist(), "prefill_seconds": m.prefill_seconds, "decode_seconds": m.decode_seconds}))
    else:  # prompts one after the other, then every sequence in the same steps
        for i, p in enumerate(prompts):
            dec.select(i)
            dec.reset()
            dec.extend(p)
        dec.continue_batch(args.max_new)
        for row in dec.generated_tokens_batch(args.max_new):
            print(json.dumps({"tokens": row.tolist()}))
    dec.close()
    ctx.close()
    return 0


def main() -> int:
    if len(sys.argv) > 1 and sys.argv[1] == "trace":
        from .trace import main as trace_main

        return trace_main(sys.argv[2:])
    ap = argparse.ArgumentParser(prog="loom_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy continuation of one or several prompts of token ids")
    g.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    g.add_argument("--tokens", action="append", required=True, help="token ids with commas between them; repeat for more sequences")
    g.add_argument("--max-new", type=int, default=16)
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    g.add_argument("--max-seq-len", type=int, default=2048)
    g.add_argument("--device", type=int, default=0)
    sub.add_parser("models", help="the registered designs")
    sub.add_parser("trace", help="replay a trace of token ids (bin/trace_run)")
    args = ap.parse_args()
    if args.command == "generate":
        return generate(args)
    from . import models

    print("\n".join(sorted(models.REGISTRY)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
