"""Replays a trace of token ids through a model: steps come as JSON lines, the logits asked for leave as files.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A step is ``{"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [...]}``.  Each
entry continues its request from what earlier steps left in the session's slot; ``want`` names places among
the entry's tokens.  ``<step>.f32`` holds their logits, little-endian fp32 in the order of the entries and of
``want``; ``done <step>`` is printed after every step.  Requests named in ``end`` give their slots back.
Single tokens of started requests run through the captured decode step, portions through prefill.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path


def replay(engine, lines, out_dir, max_tokens: int, slots: int = 4, prefill_tokens: int = 8192, report=print) -> None:
    import torch

    from .layered import Segment
    cap = max(1, min(int(max_tokens), prefill_tokens))
    session = engine.new_session(slots, max(1, int(max_tokens)), 1, cap, stop_on_end=False)
    slot_of: dict[str, int] = {}
    try:
        for line in lines:
            if not line.strip():
                continue
            step = json.loads(line)
            segments = []
            for e in step["entries"]:
                if not e["tokens"]:
                    continue
                if e["id"] not in slot_of:
                    slot_of[e["id"]] = session.acquire()
                segments.append(Segment(slot_of[e["id"]], e["tokens"], list(e.get("want", []))))
            rows = [r for r in session.step(segments) if r is not None] if segments else []
            session.poll()          # synchronises and surfaces any device-side error
            if rows:
                data = torch.cat(rows).float().cpu().numpy().astype("<f4")
                (Path(out_dir) / f"{step['step']}.f32").write_bytes(data.tobytes())
            for rid in step.get("end", []):
                if rid in slot_of:
                    session.release(slot_of.pop(rid))
            report(f"done {step['step']}")
    finally:
        session.close()


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)
    from . import build
    build.build()
    from .registry import load_model
    engine = load_model(args.model, "cuda:0", args.dtype)

    def report(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    replay(engine, sys.stdin, args.out, args.max_tokens, report=report)
    return 0
