#!/usr/bin/env python3
"""Greedy generation from a model directory (``config.json`` + safetensors) of any registered architecture.

    python -m libtbvcoll_b200.generate --model DIR --prompt 5,17,3 --prompt 9,2 --new 32 [--dtype float32]

Prompts are token ids (no tokenizer is part of the package); one JSON object per prompt is printed."""
from __future__ import annotations

import argparse
import json


def main() -> int:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="model directory, or the name of a preset with random weights")
    ap.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; repeat for a batch")
    ap.add_argument("--new", type=int, default=16, help="tokens to generate per prompt")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--max-batch", type=int, default=8)
    ap.add_argument("--eos", type=int, default=None)
    args = ap.parse_args()
    import os

    import torch

    from .engine.engine import Engine
    from .models.config import PRESETS, get_config
    from .models.registry import load_config
    from .utils.weights import SafetensorsSource
    prompts = [[int(t) for t in p.split(",")] for p in args.prompt]
    dtype = getattr(torch, args.dtype)
    if os.path.isdir(args.model):
        cfg, source = load_config(args.model), SafetensorsSource(args.model, dtype=dtype)
    elif args.model in PRESETS:
        cfg, source = get_config(args.model), None
    else:
        ap.error(f"{args.model}: neither a directory nor one of {', '.join(sorted(PRESETS))}")
    eng = Engine(cfg, device="cuda:0", source=source, dtype=dtype, max_batch=args.max_batch, max_seq_len=max(map(len, prompts)) + args.new)
    for p, o in zip(prompts, eng.generate(prompts, args.new, eos_id=args.eos)):
        print(json.dumps({"prompt": p, "tokens": o}))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
