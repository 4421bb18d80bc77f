"""Command line of the engine.

    python -m flash_attn_v100_b200.engine --model DIR --prompt 5,17,3 [--prompt ...] --max-new-tokens 32 [--dtype bfloat16]

Greedy generation from token ids with the model of a folder (config.json, model.safetensors); prompts of the same length form
one batch.  Prints one line of generated ids per prompt.
"""
from __future__ import annotations

import argparse
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m flash_attn_v100_b200.engine", description="Greedy generation from token ids.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; may be given several times")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--dtype", default=None, choices=("bfloat16", "float32"), help="default: the model family's serving type")
    ap.add_argument("--prefill-portion", type=int, default=0, help="most tokens of a prompt per pass (0: the whole prompt)")
    args = ap.parse_args(argv)
    import torch
    from . import registry
    from .runner import GenerationRunner
    prompts = [[int(t) for t in p.split(",")] for p in args.prompt]
    raw = registry.read_config(args.model)
    registry.family_of(raw).build_libraries()
    model = registry.load_model(args.model, getattr(torch, args.dtype) if args.dtype else None, config=raw)
    groups = {}
    for i, p in enumerate(prompts):
        groups.setdefault(len(p), []).append(i)
    runner = GenerationRunner(model, max_batch=max(len(g) for g in groups.values()), max_seq_len=max(groups) + args.max_new_tokens)
    results = [None] * len(prompts)
    for idx in groups.values():
        toks = runner.generate(torch.tensor([prompts[i] for i in idx]), args.max_new_tokens, prefill_portion=args.prefill_portion)
        for i, row in zip(idx, toks.tolist()):
            results[i] = row
    for row in results:
        print(",".join(str(t) for t in row))
    return 0


if __name__ == "__main__":
    sys.exit(main())
