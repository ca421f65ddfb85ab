"""Command line: `python -m jasmine_b200 generate --model DIR --prompt "5 17 3" ...` and `... trace ...`."""
from __future__ import annotations

import argparse
import sys


def generate_main(argv) -> int:
    ap = argparse.ArgumentParser(prog="jasmine_b200 generate", description="Generate tokens from token prompts by continuous batching.")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--prompt", action="append", default=[], help="token ids with spaces between them; may be repeated "
                    "(without it, one prompt per line of standard input)")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--temperature", type=float, default=0.0, help="0 = arg-max")
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--stop", type=int, action="append", default=[], help="token id that ends a sequence; may be repeated")
    ap.add_argument("--max-batch", type=int, default=8)
    ap.add_argument("--max-context", type=int, default=4096)
    ap.add_argument("--pool-pages", type=int, default=0, help="cache pages of 64 positions (0 = full contexts)")
    a = ap.parse_args(argv)
    from .generate import generate
    from .registry import load_model
    lines = a.prompt or [l for l in sys.stdin if l.strip()]
    prompts = [[int(t) for t in l.split()] for l in lines]
    model = load_model(a.model, a.dtype, max_batch=a.max_batch, max_context=a.max_context, pool_pages=a.pool_pages)
    for tokens in generate(model, prompts, a.max_new, a.temperature, a.top_k, a.top_p, a.seed, a.stop):
        print(*tokens)
    model.close()
    return 0


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else argv
    if argv and argv[0] == "generate":
        return generate_main(argv[1:])
    if argv and argv[0] == "trace":
        from .trace import main as trace_main
        return trace_main(argv[1:])
    print("usage: python -m jasmine_b200 generate|trace ... (--help for the options)", file=sys.stderr)
    return 2


if __name__ == "__main__":
    sys.exit(main())
