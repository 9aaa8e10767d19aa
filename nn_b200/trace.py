"""Replays a trace of token ids through a model and writes the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Every input line is one step as JSON:
    {"step": 7, "entries": [{"id": "x", "tokens": [11, 4, 90, 2], "want": [1, 3]}], "end": ["x"]}
`tokens` continue sequence x, `want` indexes into them: after which of them logits are to be stored. `end` closes
sequences behind the step. The wanted logits go to OUT/<step>.f32 (f32, [wanted, vocab]); 'done <step>' on
standard output acknowledges the step. The decoder holds one sequence, so one is open at a time.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

from . import api, models

DTYPES = {"bfloat16": api.BF16, "float32": api.F32}


class Replay:
    def __init__(self, decoder, stream=None):
        self.decoder, self.stream = decoder, stream
        self.live, self.pos = None, 0

    def step(self, entries, end=()):
        """Logits [wanted, vocab] of one step (None if nothing is wanted)."""
        if len(entries) > 1:
            raise ValueError(f"a step of {len(entries)} entries: this decoder holds one sequence")
        out = None
        for e in entries:
            if self.live is None:
                self.live, self.pos = e["id"], 0
            elif e["id"] != self.live:
                raise ValueError(f"request {e['id']!r} starts while {self.live!r} is live")
            want = e.get("want") or []
            if not e["tokens"]:
                continue
            order = sorted(set(want))
            got = self.decoder.extend(e["tokens"], self.pos, order, self.stream)
            self.pos += len(e["tokens"])
            if want:
                at = {w: i for i, w in enumerate(order)}
                out = got[[at[w] for w in want]]
        if self.live in end:
            self.live, self.pos = None, 0
        return out


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="a model folder or file (see nn_b200.models)")
    ap.add_argument("--dtype", default="bfloat16", choices=sorted(DTYPES))
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=4096, help="positions to make room for")
    a = ap.parse_args(argv)
    # stream 0 (the default stream) keeps the runner free of torch
    replay = Replay(models.load_model(a.model, max_seq=max(a.max_tokens, 16), act_dtype=DTYPES[a.dtype]), stream=0)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s["entries"], s.get("end") or ())
        if logits is not None:
            np.ascontiguousarray(logits, "<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    replay.decoder.backend.device_status(0)
    return 0


if __name__ == "__main__":
    sys.exit(main())
