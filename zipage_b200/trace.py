"""Replays a trace of given tokens through the serving engine and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input holds one JSON object per line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step run as one batch, each on what earlier steps left in its pages and state slot; the
logits at the wanted places are written to DIR/<step>.f32 (little-endian fp32, [wanted, vocab]);
requests in `end` then give back what they hold.  A line `done <step>` follows every step.
Nothing is sampled: the engine's own step function runs the given tokens.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

SLOTS = 4          # live requests
PAGE = 64


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of given tokens and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="most tokens that live requests hold at any time, each rounded up to a multiple of 64")
    a = ap.parse_args(argv)

    from .models import registry
    from . import build
    build.ensure(registry.kernel_part(a.model))
    import torch
    eng = registry.build_engine(a.model, dtype=getattr(torch, a.dtype), max_tokens=a.max_tokens, max_seqs=SLOTS,
                                block_size=PAGE)
    if not eng.portions:
        raise SystemExit(f"{a.model}: this architecture is served with KV compression and cannot be replayed token by token")
    vocab = eng.lm_head.shape[0]
    out_dir = Path(a.out)
    live = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        handles, counts, want = [], [], []
        for e in step["entries"]:
            toks = e["tokens"]
            if not toks or min(toks) < 0 or max(toks) >= vocab:
                raise ValueError(f"step {step['step']}: request {e['id']!r} brings no tokens or ids outside the vocabulary")
            if any(not 0 <= w < len(toks) for w in e.get("want", [])):
                raise ValueError(f"step {step['step']}: request {e['id']!r} wants places it does not bring")
            live[e["id"]] = eng.feed(toks, live.get(e["id"], -1))
            handles.append(live[e["id"]])
            counts.append(len(toks))
            want.append(e.get("want", []))
        if len(set(handles)) != len(handles):
            raise ValueError(f"step {step['step']}: a request has two entries")
        if handles:
            logits = eng.run_fed(handles, counts, want)
            if logits is not None:
                logits.cpu().numpy().astype("<f4").tofile(out_dir / f"{step['step']}.f32")
        for i in step.get("end", []):
            eng.close(live.pop(i))
        print(f"done {step['step']}", flush=True)
    return 0
