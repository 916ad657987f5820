"""Replay of a trace of token steps: given token ids run through a model's engine step by step, logits written out.

Steps come as JSON lines, ``{"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [ids]}``.
Every step's wanted logits go to ``<out>/<step>.f32`` (little-endian fp32, (wanted, vocab)), then ``done <step>`` is
printed.  Nothing is sampled; the engine's own step, slot cache and kernels run.
"""

from __future__ import annotations

import argparse
import json
import os
import sys

MAX_LIVE = 8   # requests that may hold a slot at the same time


def run(engine, lines, out_dir: str, emit=print) -> None:
    rows: dict[str, object] = {}
    for line in lines:
        if not line.strip():
            continue
        s = json.loads(line)
        entries = []
        for e in s["entries"]:
            if e["id"] not in rows:
                rows[e["id"]] = engine.new_row()
            entries.append((rows[e["id"]], e["tokens"], e["want"]))
        if entries:
            logits = engine.step(entries)
            if logits.shape[0]:
                data = logits.cpu().numpy().astype("<f4").tobytes()
                with open(os.path.join(out_dir, f"{s['step']}.f32"), "wb") as f:
                    f.write(data)
        for i in s.get("end", []):
            if i in rows:
                rows.pop(i).close()
        engine.check_device()
        emit(f"done {s['step']}", flush=True)


def add_arguments(ap: argparse.ArgumentParser) -> None:
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, default=2048, help="most tokens that live requests hold at any time")


def run_args(args) -> int:
    import torch

    from .registry import open_engine

    n = max(args.max_tokens, 1)
    engine = open_engine(args.model, dtype=getattr(torch, args.dtype), max_rows=MAX_LIVE, max_seq=n,
                         max_prefill_rows=min(max(n, 16), 4096))
    run(engine, sys.stdin, args.out)
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token steps and write the logits")
    add_arguments(ap)
    return run_args(ap.parse_args(argv))
