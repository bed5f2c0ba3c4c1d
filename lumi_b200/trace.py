"""Trace replay: feeds given token ids through a model step by step and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

DIR holds config.json and model.safetensors; the design is chosen by the config.  Steps come on standard input, one JSON
object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every entry's tokens go to the session slot its request holds (a new id takes the lowest free one) through Session.extend, the
call that prompt portions and single decode steps of every model take; requests named in "end" give their slot back.  The
wanted logits are written to OUT/<step>.f32 as little-endian fp32 [wanted, vocab], in the order of the entries, and "done
<step>" is printed after every step.  float32 widens the weights, so that products, cache and states are all fp32.
"""
from __future__ import annotations

import argparse
import fcntl
import json
import os
import sys

import numpy as np

SLOTS = 8


def _library() -> None:
    """Compiles the library where that has not been done yet (one process at a time)."""
    from . import build
    os.makedirs(build.LIBDIR, exist_ok=True)
    with open(os.path.join(build.LIBDIR, ".lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        build.build()


class Replay:
    def __init__(self, model_dir: str, dtype: str, max_tokens: int):
        from . import api
        self.model = api.NmModel.load(os.path.join(model_dir, "model.safetensors"), os.path.join(model_dir, "config.json"),
                                      widen_weights=dtype == "float32")
        self.session = self.model.init_states(SLOTS, max(max_tokens, 1))
        self.slots: dict = {}

    def slot_of(self, rid: str) -> int:
        if rid not in self.slots:
            free = [i for i in range(SLOTS) if i not in self.slots.values()]
            if not free:
                raise RuntimeError(f"more than {SLOTS} requests are live at a time")
            self.slots[rid] = free[0]
            self.session.reset([free[0]])
        return self.slots[rid]

    def step(self, step: dict):
        rows = []
        for e in step["entries"]:
            want = [int(w) for w in e.get("want", [])]
            places = sorted(set(want))
            logits = self.session.extend(e["tokens"], places, slot=self.slot_of(e["id"]))
            if want:
                rows.append(logits[[places.index(w) for w in want]])
        for rid in step.get("end", []):
            self.slots.pop(rid, None)
        return np.concatenate(rows) if rows else None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    args = ap.parse_args(argv)
    _library()
    replay = Replay(args.model, args.dtype, args.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step)
        if logits is not None:
            logits.astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        print(f"done {step['step']}", flush=True)
    return 0
