"""Replays a token trace: given ids go through a model step by step, logits come out, nothing is sampled.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps are JSON objects on standard input, one a line: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.
All entries of a step run as one batch.  The logits at the wanted places go to DIR/<step>.f32; "done <step>" follows
on standard output.  The cache pool holds N tokens and there are four sequence slots.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

from . import _lib, build
from .model import Model
from .ops import Context

SLOTS = 4
ROUND = 64


def step_rows(entries):
    """Flat places of the wanted tokens in entry order, and the same ascending without repeats plus the way back."""
    want, base = [], 0
    for e in entries:
        want += [base + int(w) for w in e.get("want", [])]
        base += len(e["tokens"])
    rows, back = np.unique(np.array(want, dtype=np.int64), return_inverse=True)
    return rows.astype(np.int32), back.reshape(-1)


class Replayer:
    def __init__(self, model):
        self.model, self.seqs = model, {}

    def step(self, entries, end):
        """Runs one step; returns the wanted logits [n, vocab] (None if nothing is wanted)."""
        entries = [e for e in entries if e["tokens"]]
        for e in entries:
            if e["id"] not in self.seqs:
                self.seqs[e["id"]] = self.model.seq_alloc()
        logits = None
        if entries:
            rows, back = step_rows(entries)
            logits = self.model.forward_batch([(self.seqs[e["id"]], e["tokens"]) for e in entries], rows)
            if logits is not None:
                logits = logits[back]
        for i in end:
            if i in self.seqs:
                self.model.seq_free(self.seqs.pop(i))
        return logits


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", type=int, default=0)
    args = ap.parse_args(argv)
    _lib.use(build.build_part("layers"))
    ctx = Context(args.device)
    n = max(ROUND, (args.max_tokens + ROUND - 1) // ROUND * ROUND)
    model = Model.from_dir(ctx, args.model, args.dtype, max_seqs=SLOTS, max_ctx=n, pool_tokens=n)
    model.finalize()
    replay = Replayer(model)
    for line in sys.stdin:
        if not line.strip():
            continue
        st = json.loads(line)
        logits = replay.step(st["entries"], st.get("end", []))
        if logits is not None:
            logits.astype("<f4").tofile(os.path.join(args.out, f"{st['step']}.f32"))
        print(f"done {st['step']}", flush=True)
    model.close()
    ctx.close()
    return 0
