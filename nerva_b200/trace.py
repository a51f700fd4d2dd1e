"""Replays a trace of given tokens through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps

Each input line is one step, {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}; the logits
at the wanted places go to OUT/<n>.f32 (little-endian float32, [wanted, vocab]) and "done <n>" is
printed.  A request is a session: the first takes the root session, others fork it (shared weights),
and a session whose request has ended serves the next one.  The tokens go through session.append,
the call start is a special case of.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

from . import registry
from .session import CudaHfDecodeSequenceSession, SmokeStatus


class TraceReplay:
    def __init__(self, folder: str, dtype: str, max_tokens: int):
        self.root = CudaHfDecodeSequenceSession(registry.load_model(folder), max(max_tokens, 2), compute=dtype)
        if self.root.status != SmokeStatus.OK:
            raise RuntimeError(f"session create {self.root.status}: {self.root.error}")
        self.idle = [self.root]
        self.live = {}   # request id -> session
        self.fresh = set()

    def _session(self, request):
        if request not in self.live:
            if self.idle:
                session = self.idle.pop()
            else:
                session = self.root.fork_shared_weights()
                if session.status != SmokeStatus.OK:
                    raise RuntimeError(f"session fork {session.status}: {session.error}")
            self.live[request] = session
            self.fresh.add(request)
        return self.live[request]

    def step(self, record: dict) -> np.ndarray:
        """Logits of the step's wanted places, in the order of the entries and of their `want`."""
        parts = [np.empty((0, self.root.config.vocab), dtype=np.float32)]
        for entry in record["entries"]:
            if not entry["tokens"]:
                continue
            session = self._session(entry["id"])
            parts.append(session.append(entry["tokens"], entry.get("want", ()), reset=entry["id"] in self.fresh))
            self.fresh.discard(entry["id"])
        for request in record.get("end", ()):
            if request in self.live:
                self.idle.append(self.live.pop(request))
                self.fresh.discard(request)
        return np.concatenate(parts)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)
    replay = TraceReplay(args.model, args.dtype, args.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        record = json.loads(line)
        logits = replay.step(record)
        if len(logits):
            logits.astype("<f4").tofile(os.path.join(args.out, f"{record['step']}.f32"))
        print(f"done {record['step']}", flush=True)
    return 0
