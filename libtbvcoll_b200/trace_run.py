"""Replays a trace of given token ids through a model, step by step, and writes the logits that the trace asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N   < steps.jsonl

A step is one JSON object on a line of standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries`` are the next tokens of each request and the offsets among them whose logits are wanted; ``end`` names requests that
are finished after the step.  All entries of a step run as one batch of ``Engine.step``.  Logits go to OUT/<step>.f32
(little-endian fp32, [wanted, vocab], in the order of the entries and offsets); ``done <step>`` is printed after every step.
Nothing is sampled.  ``--max-tokens`` sizes the cache pool: the most tokens that live requests hold at any time.  Exit code 3: the model's
architecture does not run in the requested dtype."""
from __future__ import annotations

import argparse
import json
import os
import sys

MAX_LIVE = 4          # requests live at the same time
MAX_ROWS = 8192       # token rows of one pass; a longer step runs as several


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    args = ap.parse_args(argv)

    from .models.registry import architecture_of, load_config
    cfg = load_config(args.model)
    if args.dtype not in architecture_of(cfg).dtypes:
        print(f"{cfg.name} does not run in {args.dtype}", file=sys.stderr)
        return 3

    import torch

    from .engine.engine import Engine
    from .utils.weights import SafetensorsSource
    dtype = getattr(torch, args.dtype)
    eng = Engine(cfg, device="cuda:0", source=SafetensorsSource(args.model, dtype=dtype), dtype=dtype, max_batch=MAX_LIVE,
                 max_seq_len=args.max_tokens, max_cache_tokens=args.max_tokens, prefill_chunk=max(1, min(args.max_tokens, MAX_ROWS)))
    with torch.no_grad():
        for line in sys.stdin:
            if not line.strip():
                continue
            st = json.loads(line)
            logits = eng.step([(e["id"], e["tokens"], e.get("want", ())) for e in st["entries"]], end=st.get("end", ()))
            if logits.shape[0]:
                logits.cpu().numpy().astype("<f4").tofile(os.path.join(args.out, f"{st['step']}.f32"))
            print(f"done {st['step']}", flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
