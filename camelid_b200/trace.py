"""Replays a trace: given token ids through a model, step by step, the logits at chosen places to files.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N [--max-seqs M]

Steps come on standard input, one JSON object a line:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
`entries`: the next tokens of each request and the places among them whose logits are asked for; `end`: the requests whose
slots are given back after the step.  A step in which something is wanted leaves OUT/<step>.f32: the logits in the order of
the entries and places, little-endian 32-bit floats.  After every step a line `done <step>` is printed."""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

import numpy as np


class TraceRunner:
    def __init__(self, engine):
        from .scheduler import SlotTable

        self.engine = engine
        self.slots = SlotTable(engine.cfg.max_seqs)

    def step(self, entries, end) -> np.ndarray | None:
        rows = []
        for e in entries:
            rid, tokens, want = e["id"], e["tokens"], e.get("want", [])
            if rid not in self.slots:
                self.slots.acquire(rid)
            if tokens:
                places = sorted(set(want))
                _, logits = self.engine.extend(self.slots.slot(rid), tokens, self.slots.length(rid), places)
                self.slots.advance(rid, len(tokens))
                if want:
                    rows.append(logits[[places.index(w) for w in want]])
        for rid in end:
            if rid in self.slots:
                self.slots.release(rid)
        return np.concatenate(rows) if rows else None


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True, help="the most tokens that live requests hold at any time")
    ap.add_argument("--max-seqs", type=int, default=4, help="the most requests live at any time")
    a = ap.parse_args(argv)
    from . import models

    out = Path(a.out)
    runner = TraceRunner(models.load_model(a.model, max_pos=max(1, a.max_tokens), max_seqs=a.max_seqs, dtype=a.dtype))
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = runner.step(s["entries"], s.get("end", []))
        if logits is not None:
            (out / f"{s['step']}.f32").write_bytes(np.ascontiguousarray(logits, "<f4").tobytes())
        print(f"done {s['step']}", flush=True)
    runner.engine.close()
    return 0
