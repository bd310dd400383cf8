"""Trace replay: feeds given token ids through a model step by step and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps

One JSON object a line on standard input: ``{"step": 0, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end":
[...]}``.  A step runs every entry's tokens from the cache its request's earlier steps left; ``want`` are the places
among the tokens whose logits go to ``DIR/<step>.f32`` (little-endian fp32, ``[wanted, vocab]``, entries in order), ``end`` the
requests that are over.  ``done <step>`` is printed after every step.  The model, its cache and its passes are the ones
generation uses; a missing kernel library is compiled first.  Exit code 3: the model has no fp32 form.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List

import torch


class Replay:
    """Live requests of a trace and their caches; a finished request's cache is kept for the next one."""

    def __init__(self, model, rows: int):
        self.model, self.rows = model, rows
        self.live: Dict[str, object] = {}
        self.free: List[object] = []

    def cache(self, rid):
        if rid not in self.live:
            c = self.free.pop() if self.free else self.model.make_cache(self.rows)
            c.reset()
            self.live[rid] = c
        return self.live[rid]

    def end(self, rid):
        c = self.live.pop(rid, None)
        if c is not None:
            self.free.append(c)

    def step(self, step: dict):
        """fp32 logits ``[wanted, vocab]`` on the CPU, or None when nothing is wanted."""
        out = []
        for e in step.get("entries", []):
            if not e["tokens"]:
                continue
            logits = self.model(torch.tensor(e["tokens"], dtype=torch.int32), self.cache(e["id"]), want=e.get("want", []))
            if logits is not None:
                out.append(logits[0].float().cpu())
        self.model.check_fused_error()
        for rid in step.get("end", []):
            self.end(rid)
        return torch.cat(out) if out else None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token traces through a model and write logits.")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=4096)
    a = ap.parse_args(argv)
    from . import build, load
    _, library, has_f32 = load.model_builder(load.read_config(a.model))
    if a.dtype == "float32" and not has_f32:
        print("this model has no fp32 form", file=sys.stderr)
        return 3
    build.build(libs=(library,))
    model = load.load_model(a.model, torch.device("cuda", 0), dtype=a.dtype).relayout()
    replay = Replay(model, max(64, (a.max_tokens + 63) // 64 * 64))
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step)
        if logits is not None:
            logits.numpy().astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
        print(f"done {step['step']}", flush=True)
    return 0
