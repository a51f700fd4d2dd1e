"""Generates tokens from a model folder.

    python -m nerva_b200.generate --model DIR --prompt 5,17,3 --tokens 32 [--temperature T --top-p P --top-k K
        --seed S] [--dtype bfloat16|float32] [--eos ID]

Token ids in, token ids out (one line, comma-separated): there is no tokenizer here.
"""
from __future__ import annotations

import argparse
import sys

from . import build, registry
from .session import CudaHfDecodeSequenceLoop, CudaHfDecodeSequenceSession, SmokeStatus, greedy_sampler, sampler_config


def generate(checkpoint, prompt, tokens: int, sampler=None, eos=None, compute: str = "bfloat16") -> list:
    session = CudaHfDecodeSequenceSession(checkpoint, len(prompt) + tokens, compute=compute)
    if session.status != SmokeStatus.OK:
        raise RuntimeError(f"session create {session.status}: {session.error}")
    summary, loop = CudaHfDecodeSequenceLoop.start(session, prompt, eos_token=eos, sampler=sampler)
    if loop is None:
        raise RuntimeError(f"session start {summary.status}: {summary.error}")
    out = loop.advance(tokens)
    if out.status != SmokeStatus.OK:
        raise RuntimeError(f"session advance {out.status}: {out.error}")
    session.destroy()
    return out.tokens


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m nerva_b200.generate", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompt", required=True, help="comma-separated token ids")
    ap.add_argument("--tokens", type=int, default=32)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--eos", type=int, default=None)
    args = ap.parse_args(argv)
    build.build()
    sampler = (sampler_config(args.temperature, args.top_p, args.top_k, args.seed) if args.temperature > 0.0
               else greedy_sampler())
    prompt = [int(t) for t in args.prompt.split(",")]
    print(",".join(map(str, generate(registry.load_model(args.model), prompt, args.tokens, sampler, args.eos, args.dtype))))
    return 0


if __name__ == "__main__":
    sys.exit(main())
