"""Replays a trace of token ids through a model and writes logits (the program behind bin/trace_run).

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps arrive on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

An entry carries the next tokens of one request and the places among them whose logits are asked for; ``end`` lists the
requests that are finished after the step.  A step that asks for logits writes OUT/<step>.f32, f32 little-endian rows
[wanted, vocab] in the order asked; every step is answered by a line ``done <step>``.  Requests come one after the other:
one session of N rows serves them all, through the same ``GptDecoder.decode`` as generation does.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

from . import build
from .models import load_model
from .nn import Backend, TnsrError


class TraceRunner:
    def __init__(self, model, max_tokens: int, out: str):
        self.vocab = model.config().vocab_size
        self.decoder = model.decoder_with_capacity(Backend.Cuda, 1, max(1, max_tokens))
        self.out = out
        self.live = None      # request that holds the session

    def step(self, record: dict) -> None:
        rows = []
        for entry in record["entries"]:
            if self.live is None:
                self.decoder.reset()
                self.live = entry["id"]
            elif self.live != entry["id"]:
                raise TnsrError(f"request {entry['id']!r} starts while {self.live!r} is not finished")
            if entry["tokens"]:
                logits = self.decoder.decode(entry["tokens"]).reshape(len(entry["tokens"]), self.vocab)
                rows += [logits[place] for place in entry["want"]]
        if rows:
            np.stack(rows).astype("<f4").tofile(os.path.join(self.out, f"{record['step']}.f32"))
        if self.live in record.get("end", []):
            self.decoder.reset()
            self.live = None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replays token ids through a model, step by step, and writes logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens a live request holds")
    args = ap.parse_args(argv)
    build.build()             # nothing to do unless a source is newer than the library
    runner = TraceRunner(load_model(args.model, args.dtype), args.max_tokens, args.out)
    for line in sys.stdin:
        if line.strip():
            record = json.loads(line)
            runner.step(record)
            print(f"done {record['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
