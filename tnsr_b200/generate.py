"""Generates from a model folder on the command line.

    python -m tnsr_b200.generate --model DIR --prompt "5 17 3" --max-new-tokens 32 [--temperature 0.8 --top-k 40 --seed 1]

Token ids in, token ids out (there is no tokenizer here); any architecture of the model registry works.
"""
from __future__ import annotations

import argparse
import sys

import numpy as np

from . import build
from .models import DTYPES, load_model
from .nn import Backend, TnsrError
from .session import B200Session


def sampled(model, prompt, count: int, temperature: float, top_k: int, seed: int):
    """Prompt in one step, then one token per step with the library's seeded top-k sampler (ids only leave the device)."""
    capacity = len(prompt) + count
    if capacity > model.config().max_sequence_length:
        raise TnsrError("decoder capacity must fit the model context")
    session = B200Session(model.config(), 1, capacity, logits_mode="none")
    for i, p in enumerate(model.parameters()):
        session.refresh(i, p.values())
    session.set_sampler(temperature, top_k, seed)
    ids, position, chunk = [], 0, np.asarray([prompt], dtype=np.uint32)
    for _ in range(count):
        _, new = session.decode_full(chunk, position)
        position += chunk.shape[1]
        chunk = new.reshape(1, 1)
        ids.append(int(new[0]))
    session.close()
    return ids


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="tnsr_b200.generate", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="model folder")
    ap.add_argument("--dtype", default="bfloat16", choices=sorted(DTYPES))
    ap.add_argument("--prompt", required=True, help="token ids, separated by spaces or commas")
    ap.add_argument("--max-new-tokens", type=int, default=16)
    ap.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    ap.add_argument("--top-k", type=int, default=40)
    ap.add_argument("--seed", type=int, default=0)
    args = ap.parse_args(argv)
    build.build()
    model = load_model(args.model, args.dtype)
    prompt = [int(x) for x in args.prompt.replace(",", " ").split()]
    if args.temperature > 0.0:
        ids = sampled(model, prompt, args.max_new_tokens, args.temperature, args.top_k, args.seed)
    else:
        ids = model.generate_cached(Backend.Cuda, prompt, args.max_new_tokens)[len(prompt):]
    print(" ".join(map(str, ids)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
