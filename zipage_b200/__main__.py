"""Command line of the serving engine.

    python -m zipage_b200 models                                     # registered architectures
    python -m zipage_b200 generate --model DIR --prompt 5,17,3 [...] # token ids in, token ids out
    python -m zipage_b200 trace --model DIR ...                      # as bin/trace_run

Prompts and completions are token ids (tokenizers are the caller's).
"""
from __future__ import annotations

import argparse
import json
import sys


def _generate(argv):
    ap = argparse.ArgumentParser(prog="zipage_b200 generate")
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float16", "float32"])
    ap.add_argument("--prompt", action="append", default=[], help="comma-separated token ids; repeat for a batch")
    ap.add_argument("--prompts-file", help="JSON list of token-id lists")
    ap.add_argument("--new-tokens", type=int, default=64)
    ap.add_argument("--temperature", type=float, default=1.0)
    ap.add_argument("--greedy", action="store_true")
    ap.add_argument("--eos", type=int, default=None)
    ap.add_argument("--max-tokens", type=int, default=65536, help="tokens the page pool holds")
    ap.add_argument("--max-seqs", type=int, default=8)
    ap.add_argument("--token-budget", type=int, default=8192, help="tokens of one step")
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--no-graph", action="store_true", help="decode launch by launch")
    a = ap.parse_args(argv)
    prompts = [[int(t) for t in p.split(",")] for p in a.prompt]
    if a.prompts_file:
        with open(a.prompts_file) as f:
            prompts += json.load(f)
    if not prompts:
        ap.error("no prompt given")

    from . import build
    from .models import registry
    build.ensure(registry.kernel_part(a.model))
    import torch
    from .engine.scheduler import SamplingParams, Sequence
    eng = registry.build_engine(a.model, dtype=getattr(torch, a.dtype), max_tokens=a.max_tokens, max_seqs=a.max_seqs,
                                token_budget=a.token_budget, eos=a.eos, greedy=a.greedy, graph=not a.no_graph, seed=a.seed)
    sp = SamplingParams(a.temperature, a.new_tokens, a.eos is None)
    seqs = [Sequence(p, sp) for p in prompts]
    out = eng.generate(seqs)
    for s in seqs:
        print(json.dumps(out[s._h]))
    return 0


def main(argv=None):
    argv = list(sys.argv[1:] if argv is None else argv)
    cmd = argv.pop(0) if argv else ""
    if cmd == "models":
        from .models import registry
        print("\n".join(registry.architectures()))
        return 0
    if cmd == "generate":
        return _generate(argv)
    if cmd == "trace":
        from .trace import main as trace
        return trace(argv)
    print(__doc__, file=sys.stderr)
    return 2


if __name__ == "__main__":
    sys.exit(main())
