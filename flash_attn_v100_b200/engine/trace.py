"""Trace replay: feeds given token ids through a model step by step and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A step is one JSON line {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}: every entry's request advances by its
tokens, the logits at the places `want` among them go to DIR/<n>.f32 (little-endian fp32, [wanted, vocab], in the order of the
entries), and the requests in `end` give back what they hold.  `done <n>` is printed after every step.  The requests run through
`GenerationRunner.step`, on the model, cache and kernels that serve generation; nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

_DTYPES = ("bfloat16", "float32")
EXIT_NO_SUCH_TYPE = 3      # the model does not run in the type asked for
MAX_REQUESTS = 16          # live requests


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay given tokens through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=_DTYPES)
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)
    import torch
    from ..kv_cache import BLOCK_SIZE
    from . import registry
    from .runner import GenerationRunner
    raw = registry.read_config(args.model)
    family = registry.family_of(raw)
    dtype = getattr(torch, args.dtype)
    if dtype not in family.dtypes:
        print(f"{family.architecture} does not run in {args.dtype}", file=sys.stderr)
        return EXIT_NO_SUCH_TYPE
    family.build_libraries()
    model = registry.load_model(args.model, dtype, config=raw)
    blocks = (args.max_tokens + BLOCK_SIZE - 1) // BLOCK_SIZE + MAX_REQUESTS      # every request may leave a block part filled
    runner = GenerationRunner(model, max_batch=MAX_REQUESTS, max_seq_len=max(args.max_tokens, 1), num_blocks=blocks)
    live = set()
    for line in sys.stdin:
        if not line.strip():
            continue
        rec = json.loads(line)
        for e in rec["entries"]:
            if e["id"] not in live:
                runner.start(e["id"])
                live.add(e["id"])
        logits = runner.step([(e["id"], e["tokens"], e["want"]) for e in rec["entries"]]) if rec["entries"] else []
        runner.check_errors()
        if any(e["want"] for e in rec["entries"]):
            data = torch.cat(logits).float().cpu().contiguous().numpy().astype("<f4")
            path = os.path.join(args.out, f"{rec['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(data.tobytes())
            os.replace(path + ".part", path)
        for r in rec["end"]:
            runner.finish(r)
            live.discard(r)
        print(f"done {rec['step']}", flush=True)
    return 0
