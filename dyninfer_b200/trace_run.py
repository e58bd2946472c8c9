"""Replays a token trace through a model, step by step, and writes logits (nothing is sampled).

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

The session, its cache and its step calls are the ones generation uses. Steps come as one JSON object a
line on standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

`entries` gives each request's next tokens and the places among them whose logits are wanted, `end` the
requests that are finished after the step. A step with wanted places writes `<step>.f32` into --out
(little-endian f32 rows of `vocab` logits, in the order of the entries and of `want`); every step then prints
`done <step>`. The library is built first if it is not there.

`bfloat16` serves the model as usual (16-bit operands where the serving kernels use them, bf16 cache);
`float32` keeps the cache in f32 and multiplies in f32 throughout.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


class Replay:
    """Requests of a trace in the slots of one batched session. A slot is handed on when its request ends;
    the next request starts it over."""

    def __init__(self, session, slots: int):
        self.session, self.free, self.slot_of, self.started = session, list(range(slots)), {}, set()

    def run(self, step: dict):
        rows = []
        for e in step["entries"]:
            rid = e["id"]
            if rid not in self.slot_of:
                if not self.free:
                    raise RuntimeError(f"no free slot for request {rid}")
                self.slot_of[rid] = self.free.pop(0)
            slot = self.slot_of[rid]
            rows.append(self.session.extend_slot(slot, e["tokens"], e.get("want", ()), restart=rid not in self.started))
            self.started.add(rid)
        for rid in step.get("end", ()):
            if rid in self.slot_of:
                self.free.append(self.slot_of.pop(rid))
                self.started.discard(rid)
        rows = [r for r in rows if len(r)]
        return np.concatenate(rows) if rows else None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--slots", type=int, default=2, help="requests that may be live at once")
    args = ap.parse_args(argv)

    from . import build
    from .runtime import ModelLoader, SessionConfig
    build.build()
    cap = max(1, args.max_tokens)
    f32 = args.dtype == "float32"
    model = ModelLoader().load(args.model, max_kv=cap, kv_dtype="f32" if f32 else "bf16",
                               compute="f32" if f32 else "serve")
    with model.create_batched_session(SessionConfig(max_sequence_length=cap, batch_size=args.slots)) as session:
        replay = Replay(session, args.slots)
        for line in sys.stdin:
            if not line.strip():
                continue
            step = json.loads(line)
            logits = replay.run(step)
            if logits is not None:
                logits.astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
            print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
