"""Replays a trace: token ids fed step by step through a model, logits written where they are asked for.

Steps arrive as JSON lines on standard input:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
An entry continues its request where the last step left it; a request in "end" is given back after the
step.  A step that wants logits writes OUT/<step>.f32 (little-endian fp32, [wanted, vocab]); every step
prints "done <step>".
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


class Replay:
    """The engine holds one sequence, so one request is live at a time."""

    def __init__(self, engine):
        self.engine = engine
        self.live: str | None = None
        self.pos = 0

    def step(self, entries: list[dict], end: list[str]) -> np.ndarray:
        rows = []
        for e in entries:
            tokens, want = e["tokens"], e.get("want", [])
            if not tokens:
                if want:
                    raise ValueError(f"request {e['id']!r}: logits are asked for without tokens")
                continue
            if self.live is None:
                self.live, self.pos = e["id"], 0
                self.engine.ResetKV()
            elif self.live != e["id"]:
                raise ValueError(f"request {e['id']!r} starts before {self.live!r} has ended")
            # the engine takes ascending places; the trace may name them in any order
            places = sorted(set(want))
            got = self.engine.Forward(tokens, self.pos, places)
            rows += [got[places.index(w)] for w in want]
            self.pos += len(tokens)
        for i in end:
            if i == self.live:
                self.live = None
        return np.stack(rows) if rows else np.empty((0, self.engine.cfg.vocab), np.float32)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens live requests hold at any time (sizes the cache)")
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)

    from . import _lib, registry
    arch, _ = registry.read_config(a.model)
    _lib.provision(arch.family)
    engine = registry.load_model(a.model, dtype=a.dtype, max_seq=a.max_tokens or None, device=a.device)
    replay = Replay(engine)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s.get("entries", []), s.get("end", []))
        if len(logits):
            np.ascontiguousarray(logits, dtype="<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    engine.close()
    return 0
