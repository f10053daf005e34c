"""Replay of a step trace: feeds given token ids through a model step by step and writes the logits that were asked for.
Nothing is sampled.  The steps run through the engine's own ragged forward, page pool, block tables and recurrent slots
(`CausalLm.step_at`); this module only reads the trace and keeps one cache per live request.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A step is one JSON line {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  `want` lists places among the
entry's tokens; their logits go to OUT/<step>.f32 as little-endian f32 rows [wanted, vocab], entry by entry.  `end` lists
requests whose pages and slot are given back after the step.  "done <step>" is printed after every step.
"""
import argparse
import json
import os
import sys

import numpy as np

PAGE = 16        # tokens per page
MAX_LIVE = 4     # requests that hold a block-table row and a recurrent slot at a time


def replay(model, pool, steps, emit):
    """Runs the steps (an iterable of dicts); emit(step number, rows or None) after each."""
    from . import engine as eng

    live = {}
    try:
        for st in steps:
            seqs, wants = [], []
            for e in st["entries"]:
                if e["id"] not in live:
                    live[e["id"]] = eng.PagedKvCache(pool)
                seqs.append((np.asarray(e["tokens"], np.int32), live[e["id"]]))
                wants.append(list(e.get("want", [])))
            rows = None
            if seqs:
                rows, _ = model.step_at(seqs, wants)
            for rid in st.get("end", []):
                if rid in live:
                    live.pop(rid).free()
            emit(st["step"], rows if any(wants) else None)
    finally:
        for c in live.values():
            c.free()


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", dest="max_tokens", type=int, required=True, help="tokens the page pool holds")
    args = ap.parse_args(argv)

    from . import build

    build.build()
    from . import _lib, engine as eng

    ctx = _lib.Context(0)
    model = eng.CausalLm.open(ctx, args.model, f32=args.dtype == "float32")
    pages = max((args.max_tokens + PAGE - 1) // PAGE, 1)
    pool = eng.BlockPool(ctx, model, PAGE, pages, MAX_LIVE, pages)

    def emit(step, rows):
        if rows is not None:
            rows.astype("<f4", copy=False).tofile(os.path.join(args.out, f"{step}.f32"))
        print(f"done {step}", flush=True)

    replay(model, pool, (json.loads(line) for line in sys.stdin if line.strip()), emit)
    pool.free()
    model.free()
    ctx.close()
    return 0
