"""Replays a token trace through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A step is one line of standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every entry carries the next tokens of a request (its first entry admits it); all entries of a step run as one pass of the
family's runner, the pass the serving engine uses, over its paged pool of N cache positions and four state slots.  `want`
names the places among an entry's tokens whose logits are written to DIR/<step>.f32 (little-endian fp32 [wanted, vocab], in
the order of the entries).  `end` lists requests whose pages and slot are given back after the step.  After every step the
line "done <step>" is printed.  Nothing is sampled.  Exit status 3: the model's family does not run in the asked dtype.

The first run in a checkout compiles the host runtime and the kernels of the model's family.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

SLOTS = 4
PAGE = 64
MAX_ROWS = 2048              # rows of one pass; a longer step is carried out in several


class Replay:
    def __init__(self, model_dir: str, dtype: str, max_tokens: int):
        import torch

        from ..loaders.family_io import load_family, runner_for

        pool = -(-max_tokens // PAGE) * PAGE
        model = load_family(model_dir, "cuda", getattr(torch, dtype))
        self.runner = runner_for(model, min(MAX_ROWS, max(pool, SLOTS)), SLOTS, pool, "cuda", pool)
        if not self.runner.mixed_runs:
            raise SystemExit(f"{type(model).__name__} has no mixed pass")
        self.free = list(range(SLOTS))
        self.slot = {}

    def step(self, entries, end):
        """-> fp32 logits [wanted, vocab] on the host, or None when nothing is wanted."""
        from ..ops import core as ops

        batch = []
        for e in entries:
            if e["id"] not in self.slot:
                if not self.free:
                    raise RuntimeError("more than four live requests")
                self.slot[e["id"]] = self.free.pop(0)
            batch.append((self.slot[e["id"]], list(e["tokens"]), list(e["want"])))
        logits = None
        if batch:
            out = self.runner.step(batch)
            if any(want for _, _, want in batch):
                logits = out.float().cpu()
            ops.check_status()
        for rid in end:
            s = self.slot.pop(rid, None)
            if s is not None:
                self.runner.reset(s)
                self.free.append(s)
        return logits


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    a = ap.parse_args(argv)
    from .. import build
    from ..loaders import PUBLISHED

    with open(os.path.join(a.model, "config.json")) as f:
        cfg = json.load(f)
    family = str(cfg.get("architecture", "")).lower()
    if a.dtype == "float32" and family not in PUBLISHED:
        print("this model's family does not run in float32", file=sys.stderr)
        return 3
    kernels = build.ensure(family)
    from ..ops import _lib

    _lib.use(kernels)
    replay = Replay(a.model, a.dtype, a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s.get("entries", []), s.get("end", []))
        if logits is not None:
            part = os.path.join(a.out, f".{s['step']}.part")
            logits.numpy().astype("<f4", copy=False).tofile(part)
            os.replace(part, os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    return 0
