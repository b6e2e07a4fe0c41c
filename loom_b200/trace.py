"""Replays a trace of token ids through a model and writes the logits it asks for (`bin/trace_run`).

Steps come as JSON lines on standard input: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  Every request
holds one of the decoder's sequences from its first tokens until it ends; a step appends its tokens from the state that
earlier steps left (`Decoder.extend`, the call that prompts and decoding go through).  For a step with wanted places
<out>/<step>.f32 receives the logits, then "done <step>" is printed.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

SEQUENCES = 8  # requests alive at a time


class Sequences:
    """Which request holds which sequence of a decoder."""

    def __init__(self, decoder):
        self.decoder = decoder
        self.lane_of: dict = {}
        self.free = list(range(decoder.batch))

    def select(self, request: str):
        if request not in self.lane_of:
            if not self.free:
                raise RuntimeError("more than %d requests at a time" % self.decoder.batch)
            self.lane_of[request] = self.free.pop(0)
            self.decoder.select(self.lane_of[request])
            self.decoder.reset()
        else:
            self.decoder.select(self.lane_of[request])

    def end(self, request: str):
        lane = self.lane_of.pop(request, None)
        if lane is not None:
            self.free.append(lane)


def run(decoder, lines, out_dir: str, echo) -> None:
    seqs = Sequences(decoder)
    for line in lines:
        line = line.strip()
        if not line:
            continue
        step = json.loads(line)
        rows = []
        for entry in step["entries"]:
            seqs.select(entry["id"])
            want = entry.get("want", [])
            if not entry["tokens"]:
                continue
            places = sorted(set(want))
            logits = decoder.extend(entry["tokens"], places)
            if want:
                rows.append(logits[[places.index(w) for w in want]])
        if rows:
            np.concatenate(rows).astype("<f4").tofile(os.path.join(out_dir, "%d.f32" % step["step"]))
        for request in step.get("end", []):
            seqs.end(request)
        echo("done %d" % step["step"])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="feed given token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=2048, help="the most tokens that live requests hold")
    args = ap.parse_args(argv)
    from . import build

    build.build()
    from . import Context, models

    ctx = Context(0)
    decoder = models.load(ctx, args.model, args.dtype, max_seq_len=max(args.max_tokens, 2), batch=SEQUENCES)

    def echo(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    run(decoder, sys.stdin, args.out, echo)
    decoder.close()
    ctx.close()
    return 0
