"""``bin/trace_run``: replays given token ids through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come as JSON lines on standard input: ``{"step": 0, "entries": [{"id": "a", "tokens": [...], "want": [...]}],
"end": []}``.  A step feeds a request's next tokens to the model from the cache earlier steps left; the logits at the places
``want`` names go to ``DIR/<step>.f32`` (little-endian f32, ``[wanted, vocab]``), then ``done <step>`` is printed.  ``end``
gives a finished request's cache back.  Nothing is sampled.

The engine serves one sequence at a time, so the requests of a trace follow one another.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path


class TraceError(RuntimeError):
    pass


class Replay:
    """The requests of a trace over one model handle."""

    def __init__(self, model):
        self.model, self.live = model, None

    def step(self, step: dict) -> bytes:
        import numpy as np
        out = []
        for entry in step.get("entries", []):
            if self.live is None:
                self.model.reset()
                self.live = entry["id"]
            elif self.live != entry["id"]:
                raise TraceError(f"request {entry['id']!r} begins while {self.live!r} is live")
            want = list(entry.get("want", []))
            rows = sorted(set(want))
            logits = self.model.prefill_rows(entry["tokens"], rows)
            out.append(logits[[rows.index(w) for w in want]])
        for name in step.get("end", []):
            if name == self.live:
                self.model.reset()
                self.live = None
        return np.concatenate(out).astype("<f4").tobytes() if out else b""


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replays token ids through a model and writes logits.")
    ap.add_argument("--model", required=True, type=Path, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, type=Path, help="folder the logits are written to")
    ap.add_argument("--max-tokens", required=True, type=int, help="tokens a live request holds at most: sizes the cache")
    args = ap.parse_args(argv)
    from . import _lib, build, registry
    opened = registry.open_model(args.model)
    if args.dtype not in opened.dtypes:
        print(f"the {opened.family} family does not serve {args.dtype}", file=sys.stderr)
        return 3
    if opened.family == "dense":
        build.build()
        _lib.load()
    else:
        _lib.load(build.ensure("layered"))
    model = opened.load(max(1, args.max_tokens), args.dtype)
    replay = Replay(model)
    args.out.mkdir(parents=True, exist_ok=True)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        data = replay.step(step)
        if data:
            (args.out / f"{step['step']}.f32").write_bytes(data)
        print(f"done {step['step']}", flush=True)
    model.close()
    return 0
