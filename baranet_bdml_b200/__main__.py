"""Command line:

    python -m baranet_bdml_b200 generate --model DIR [--dtype bfloat16] [--max-new-tokens N] --prompt "5 17 3" [--prompt ...]
    python -m baranet_bdml_b200 trace --model DIR --out DIR < steps.jsonl

`generate` continues prompts of token ids greedily and prints one line of ids per prompt."""
from __future__ import annotations

import argparse
import sys


def generate(argv) -> int:
    ap = argparse.ArgumentParser(prog="generate")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--max-new-tokens", type=int, default=50)
    ap.add_argument("--prompt", action="append", required=True, help="token ids, separated by spaces or commas")
    a = ap.parse_args(argv)
    from . import registry
    prompts = [[int(t) for t in p.replace(",", " ").split()] for p in a.prompt]
    model = registry.load_model(a.model, a.dtype)
    for row in model.generate(prompts, a.max_new_tokens):
        print(*row)
    model.status()
    return 0


def main(argv=None) -> int:
    argv = list(sys.argv[1:] if argv is None else argv)
    if argv[:1] == ["generate"]:
        return generate(argv[1:])
    if argv[:1] == ["trace"]:
        from .trace import main as trace
        return trace(argv[1:])
    print(__doc__, file=sys.stderr)
    return 2


if __name__ == "__main__":
    sys.exit(main())
