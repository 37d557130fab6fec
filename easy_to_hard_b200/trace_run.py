"""Trace replay on the engine: one JSON line on standard input is one step; the logits it asks for
go to files. There is no sampler in the loop.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

    {"step": 7, "entries": [{"id": "s1", "tokens": [11, 4, 90], "want": [2]}], "end": ["s1"]}

``tokens`` continue the sequence ``id`` (opened at its first appearance), ``want`` indexes into
them, ``end`` closes sequences after the step. ``OUT/<step>.f32`` receives the fp32 little-endian
logits, one row per wanted place; ``done <step>`` on standard output acknowledges every step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Optional, Sequence

import torch

SLOTS = 8      # sequences that may be live at a time


def main(argv: Optional[Sequence[str]] = None, lines=None) -> int:
    ap = argparse.ArgumentParser(description="Replay recorded token ids on the engine and dump logits.")
    ap.add_argument("--model", required=True, help="checkpoint folder")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="positions the cache is built for")
    a = ap.parse_args(argv)
    from .models.engine import get_engine
    from .models.hybrid import config_in, hybrid_config, kernel_sources, load_hybrid
    from .ops import _lib
    cfg = config_in(a.model)
    if cfg is not None:
        _lib.build_only(kernel_sources(hybrid_config(cfg)))
    model = load_hybrid(a.model, "cuda", getattr(torch, a.dtype))
    eng = get_engine(model, SLOTS, max(a.max_tokens, 1), use_graph=False)
    for line in (sys.stdin if lines is None else lines):
        if not line.strip():
            continue
        req = json.loads(line)
        for e in req["entries"]:
            if e["id"] not in eng.cache:
                eng.open(e["id"])
        logits = eng.step([(e["id"], e["tokens"], e["want"]) for e in req["entries"]])
        data = logits.cpu().numpy().astype("<f4")
        code = _lib.read_status()
        if code:
            raise RuntimeError(f"a kernel reported status {code}")
        if len(data):
            tmp = os.path.join(a.out, f"{req['step']}.f32.part")
            with open(tmp, "wb") as fh:
                fh.write(data.tobytes())
            os.replace(tmp, os.path.join(a.out, f"{req['step']}.f32"))
        for key in req.get("end", []):
            if key in eng.cache:
                eng.close(key)
        print(f"done {req['step']}", flush=True)
    return 0
