"""Replay of token traces: given token ids go through the engine step by step, chosen logits are written to files.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Standard input holds one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

An entry appends tokens to request ``id``; ``want`` lists the places among them whose logits are asked for; ``end`` lists the
requests that are over after the step.  Logits go to ``<out>/<step>.f32`` (little-endian float32, [wanted, vocab]) when any are
wanted, and ``done <step>`` is printed after every step.  The model is chosen by ``config.json``; the tokens take the path of
generation (``Engine``'s chunk path, decode step, caches and states).  The engine holds one sequence at a time.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import List, Optional

DTYPES = {"bfloat16": "bf16", "float32": "fp32"}


class TraceError(RuntimeError):
    pass


class TraceRunner:
    """Maps the requests of a trace onto an engine with ``extend`` and ``reset``."""

    def __init__(self, engine, out_dir: str):
        self.engine, self.out_dir = engine, out_dir
        self.active: Optional[str] = None

    def step(self, record: dict) -> None:
        rows = []
        for entry in record.get("entries", ()):
            rid = str(entry["id"])
            if self.active is None:
                self.engine.reset()
                self.active = rid
            elif self.active != rid:
                raise TraceError(f"request {rid} starts while {self.active} is running: the engine holds one sequence")
            want = [int(w) for w in entry.get("want", ())]
            order = sorted(set(want))
            logits = self.engine.extend([int(t) for t in entry["tokens"]], order)
            if want:
                rows.append(logits[[order.index(w) for w in want]] if want != order else logits)
        if rows:
            data = b"".join(r.float().cpu().contiguous().numpy().astype("<f4").tobytes() for r in rows)
            path = os.path.join(self.out_dir, f"{record['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(data)
            os.replace(path + ".part", path)
        for rid in record.get("end", ()):
            if str(rid) == self.active:
                self.engine.reset()
                self.active = None


def build_engine(model: str, dtype: str, max_tokens: int):
    import torch
    from ..models.registry import resolve_checkpoint_model
    from .engine import Engine, StackSpec
    spec = resolve_checkpoint_model(model)
    if not isinstance(spec, StackSpec):
        raise TraceError(f"{spec.name} runs in speculative rounds only and cannot be fed step by step")
    torch.cuda.set_device(0)
    return Engine.build(spec, capacity=max(64, max_tokens), target_ckpt=model, device=torch.device("cuda", 0), dtype=dtype)


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a token trace from standard input and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=sorted(DTYPES), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens a live request holds")
    a = ap.parse_args(argv)
    os.makedirs(a.out, exist_ok=True)
    engine = build_engine(a.model, DTYPES[a.dtype], a.max_tokens)
    runner = TraceRunner(engine, a.out)
    try:
        for line in sys.stdin:
            if line.strip():
                record = json.loads(line)
                runner.step(record)
                print(f"done {record['step']}", flush=True)
    finally:
        engine.close()
    return 0
