"""Trace replay: batches of tokens decided elsewhere go through a model, chosen logits come out.

    bin/trace_run --model FOLDER --dtype bfloat16 --out FOLDER --max-tokens 4096 < batches.jsonl

Each input line is one engine step, a JSON object:

    {"step": 7, "entries": [{"id": "chat-1", "tokens": [11, 4], "want": [1]}, {"id": "doc", "tokens": [90]}], "end": ["doc"]}

`entries` are the requests of the batch with the tokens they continue with (an unknown id is a new request), `want`
the indices into those tokens whose logits are written, `end` the requests to drop once the step has run; their cache
pages and slots serve later requests.  A step that wants logits leaves <step>.f32 in the output folder: raw
little-endian f32 rows of the vocabulary's length, entry by entry.  "done <step>" on standard output acknowledges every
step.  No token is drawn.

The page pool is made for --max-tokens cached tokens over all live requests (four at most).  Exit code 3 says that the
model has no float32 path.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

LIVE_REQUESTS = 4


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Run prepared token batches through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="cached tokens the page pool is made for")
    args = ap.parse_args(argv)

    from . import build

    build.build()
    from .models import PAGE_TOKENS, Limits, UnsupportedDtype, load_model
    from .serving import TokenFeeder

    pages = max((args.max_tokens + PAGE_TOKENS - 1) // PAGE_TOKENS, 1)
    try:
        loaded = load_model(args.model, args.dtype, Limits(max_rows=pages * PAGE_TOKENS, max_reqs=LIVE_REQUESTS, max_seqs=LIVE_REQUESTS))
    except UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return 3

    import torch

    feeder = TokenFeeder(loaded, pages)
    with torch.cuda.stream(torch.cuda.Stream()):  # a stream of its own: decode-only steps replay as CUDA graphs
        for line in sys.stdin:
            if not line.strip():
                continue
            step = json.loads(line)
            logits = feeder.step([(e["id"], e["tokens"], e.get("want", ())) for e in step["entries"]])
            if len(logits):
                logits.astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
            for name in step.get("end", ()):
                feeder.end(name)
            print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
