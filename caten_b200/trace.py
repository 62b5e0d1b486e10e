"""Replays a trace of token portions through a stored model and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR [--max-tokens N]

Reads one JSON object a line from standard input,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

feeds the entry's tokens to its request, writes the logits at the wanted places of the portion to
OUT/<step>.f32 (little-endian fp32, [wanted, vocab]; no file when nothing is wanted) and prints
"done <step>".  A request's first portion starts a new sequence; "end" names requests that are
finished.  Requests come one after the other.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

from .registry import load_model
from .runtime import B200Runtime

PRECISIONS = {"bfloat16": "bf16", "float32": "fp32"}


class Replay:
    """The live request and where it stands."""

    def __init__(self, model):
        self.model, self.live, self.pos = model, None, 0

    def step(self, entries, end):
        """Logits [wanted, vocab] of one step, or None when nothing is wanted."""
        out = []
        if len(entries) > 1:
            raise ValueError("a step has at most one entry")
        for e in entries:
            if self.live is None:
                self.live, self.pos = e["id"], 0
            elif self.live != e["id"]:
                raise ValueError(f"request {e['id']!r} starts before {self.live!r} has ended")
            tokens = np.asarray(e["tokens"], np.int64)
            if tokens.size:
                logits, _ = self.model.step(tokens[None], self.pos, e["want"])
                self.pos += tokens.size
                if len(e["want"]):
                    out.append(logits[0])
        if self.live is not None and self.live in end:
            self.live = None
        return np.concatenate(out, axis=0) if out else None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=sorted(PRECISIONS))
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=4096, help="longest sequence")
    args = ap.parse_args(argv)
    with B200Runtime(0) as rt:
        model = load_model(args.model, rt, max_seq_len=max(1, args.max_tokens), batch=1, precision=PRECISIONS[args.dtype])
        replay = Replay(model)
        for line in sys.stdin:
            if not line.strip():
                continue
            s = json.loads(line)
            logits = replay.step(s["entries"], s["end"])
            if logits is not None:
                np.ascontiguousarray(logits, dtype="<f4").tofile(os.path.join(args.out, f"{s['step']}.f32"))
            print(f"done {s['step']}", flush=True)
        model.close()
    return 0
