"""Command line.

    python -m dmlx_b200 generate --model DIR --prompt 101,7,42 --prompt 9,30 --max-new-tokens 32 [--temperature 0.8 --top-k 50]
    python -m dmlx_b200 trace --model DIR --out DIR --max-tokens N < steps
    python -m dmlx_b200 build
"""
from __future__ import annotations

import argparse
import json
import sys


def _token_list(text: str):
    return [int(t) for t in text.replace(",", " ").split()]


def _generate(argv) -> int:
    ap = argparse.ArgumentParser(prog="dmlx_b200 generate", description="Generate from token ids with a model folder.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--prompt", action="append", type=_token_list, required=True, help="token ids, separated by commas; may be given several times")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--stop", type=_token_list, default=[], help="token ids that end a request")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--temperature", type=float, default=0.0, help="0 = greedy")
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--prefill-chunk", type=int, default=512)
    ap.add_argument("--prefix-sharing", action="store_true", help="requests take over the prompt pages a live request already holds")
    a = ap.parse_args(argv)
    from .models import Limits, UnsupportedDtype, load_model
    from .serving import generate

    n = min(len(a.prompt), 256)
    try:
        loaded = load_model(a.model, a.dtype, Limits(max_rows=max(2048, n + a.prefill_chunk), max_reqs=n, max_seqs=n))
    except UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return 3
    out = generate(loaded, a.prompt, a.max_new_tokens, stop_tokens=a.stop, temperature=a.temperature, top_k=a.top_k, top_p=a.top_p,
                   seed=a.seed, prefill_chunk=a.prefill_chunk, prefix_sharing=a.prefix_sharing)
    for tokens in out:
        print(json.dumps(tokens))
    return 0


def main() -> int:
    argv = sys.argv[1:]
    command = argv[0] if argv else ""
    if command == "build":
        from . import build

        print(build.build(force="--force" in argv))
        return 0
    if command == "trace":
        from .replay import main as replay

        return replay(argv[1:])
    if command == "generate":
        from . import build

        build.build()
        return _generate(argv[1:])
    print(__doc__.strip(), file=sys.stderr)
    return 2


if __name__ == "__main__":
    sys.exit(main())
