"""Command line: ``python -m vui_b200 <command>``.

    info      the architecture and sizes of a checkpoint
    generate  continue prompts of token ids with a token model (one JSON list of new ids per prompt)
    trace     replay a trace of token steps and write the logits
"""

from __future__ import annotations

import argparse
import json
import sys

from . import trace


def _ids(text: str) -> list[int]:
    return [int(t) for t in text.replace(",", " ").split()]


def _info(args) -> int:
    from .registry import architecture_of, load_model

    m = load_model(args.model, device="cpu")
    n = sum(t.numel() for t in m.sd.values())
    print(json.dumps({"architecture": architecture_of(args.model), "parameters": n, "tensors": len(m.sd)}))
    return 0


def _generate(args) -> int:
    import torch

    from .registry import open_engine
    from .token_engine import TokenEngine, TokenGenConfig

    prompts = [_ids(p) for p in args.prompt_ids]
    if args.prompts_file:
        with open(args.prompts_file) as f:
            prompts += [_ids(line) for line in f if line.strip()]
    if not prompts or not all(prompts):
        print("no prompt: give --prompt-ids or --prompts-file", file=sys.stderr)
        return 2
    engine = open_engine(args.model, dtype=getattr(torch, args.dtype), max_rows=min(args.max_rows, len(prompts)),
                         max_seq=args.max_seq, seed=args.seed)
    if not isinstance(engine, TokenEngine):
        print("generate takes token models", file=sys.stderr)
        return 2
    cfg = TokenGenConfig(max_new_tokens=args.max_new_tokens, temperature=args.temperature, top_k=args.top_k,
                         rep_penalty=args.rep_penalty, rep_window=args.rep_window, stop_ids=tuple(args.stop_id))
    for ids in engine.generate(prompts, cfg):
        print(json.dumps(ids), flush=True)
    engine.check_device()
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="vui_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    p = sub.add_parser("info", help="architecture and sizes of a checkpoint")
    p.add_argument("--model", required=True)
    p.set_defaults(fn=_info)
    p = sub.add_parser("generate", help="continue prompts of token ids")
    p.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    p.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    p.add_argument("--prompt-ids", action="append", default=[], help="token ids, separated by commas or spaces; repeatable")
    p.add_argument("--prompts-file", help="one prompt of token ids per line")
    p.add_argument("--max-new-tokens", type=int, default=64)
    p.add_argument("--temperature", type=float, default=1.0)
    p.add_argument("--top-k", type=int, default=1, help="1: greedy, 0: the whole distribution")
    p.add_argument("--rep-penalty", type=float, default=1.0)
    p.add_argument("--rep-window", type=int, default=0)
    p.add_argument("--stop-id", type=int, action="append", default=[])
    p.add_argument("--max-rows", type=int, default=64, help="most sequences in flight")
    p.add_argument("--max-seq", type=int, default=None)
    p.add_argument("--seed", type=int, default=0)
    p.set_defaults(fn=_generate)
    p = sub.add_parser("trace", help="replay a trace of token steps")
    trace.add_arguments(p)
    p.set_defaults(fn=trace.run_args)
    args = ap.parse_args(argv)
    return args.fn(args)


if __name__ == "__main__":
    sys.exit(main())
