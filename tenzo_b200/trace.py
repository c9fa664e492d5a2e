"""Replay of a token trace through a model, step by step (bin/trace_run): given token ids in, logits out, no sampling.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps

Every input line is one step, a JSON object

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}

`entries` brings the next tokens of a request and the places among them whose logits are wanted, `end` the requests that
are finished after the step. Logits go to OUT/<step>.f32 (little-endian fp32, [wanted][vocab]); a line `done <step>`
follows every step. The tokens go through Engine.forward: one token of a request is the engine's decode step, several
are a prefill portion.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path


class Replay:
    """Requests on the engine's slots: a request takes a slot with its first tokens and gives it back when it ends."""

    def __init__(self, engine):
        self.engine = engine
        self.slots: dict[str, int] = {}
        self.free = list(range(engine.batch))[::-1]

    def step(self, step: dict):
        import numpy as np
        rows = []
        for e in step["entries"]:
            rid = e["id"]
            if rid not in self.slots:
                if not self.free:
                    raise RuntimeError("more live requests than the engine has slots")
                self.slots[rid] = self.free.pop()
                self.engine.reset_seq(self.slots[rid])
            if e["tokens"]:
                want = e.get("want", [])
                order = sorted(set(want))
                got = self.engine.forward(e["tokens"], order, seq=self.slots[rid])
                rows += [got[order.index(w)] for w in want]
        for rid in step.get("end", []):
            slot = self.slots.pop(rid, None)
            if slot is not None:
                self.engine.reset_seq(slot)
                self.free.append(slot)
        return np.stack(rows).astype("<f4") if rows else None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a token trace through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and the model's weights")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16", help="arithmetic of activations and matrix products")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens that live requests hold at any time (states here have a fixed size)")
    a = ap.parse_args(argv)
    from .engine import Engine
    out = Path(a.out)
    with Engine.open(a.model, compute=a.dtype) as engine:
        replay = Replay(engine)
        for line in sys.stdin:
            if not line.strip():
                continue
            step = json.loads(line)
            logits = replay.step(step)
            if logits is not None:
                logits.tofile(out / f"{step['step']}.f32")
            print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
