"""Command line:

    python -m nativebit_b200 generate --model DIR --prompt 5,17,3 --tokens 32 [--dtype bfloat16|float32] [--context N]
    python -m nativebit_b200 trace --model DIR --dtype ... --out DIR --max-tokens N      (see nativebit_b200.trace)
    python -m nativebit_b200 models

`generate` prints the greedy continuation's token ids, one comma-separated line per prompt (several --prompt options of one
length run as a batch).  A model folder holds config.json, whose "architecture" names the family, and the weights."""
from __future__ import annotations

import argparse
import sys


def _generate(argv: list[str]) -> int:
    ap = argparse.ArgumentParser(prog="nativebit_b200 generate")
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompt", required=True, action="append", help="comma-separated token ids")
    ap.add_argument("--tokens", type=int, default=32, help="tokens to generate")
    ap.add_argument("--dtype", default="bfloat16", choices=("bfloat16", "float32"))
    ap.add_argument("--context", type=int, default=4096)
    args = ap.parse_args(argv)
    prompts = [[int(t) for t in p.split(",")] for p in args.prompt]
    if len({len(p) for p in prompts}) != 1:
        ap.error("the prompts of a batch have one length")
    from . import registry
    registry.build_for(registry.read_config(args.model))
    import torch
    model = registry.load_model(args.model, args.dtype, args.context)
    session = registry.open_session(model, len(prompts))
    out = session.generate(torch.tensor(prompts, dtype=torch.long, device=session.dev), args.tokens)
    session.check()
    for row in out.tolist():
        print(",".join(str(t) for t in row))
    return 0


def main(argv: list[str] | None = None) -> int:
    argv = sys.argv[1:] if argv is None else argv
    cmd = argv[0] if argv else ""
    if cmd == "generate":
        return _generate(argv[1:])
    if cmd == "trace":
        from .trace import main as trace
        return trace(argv[1:])
    if cmd == "models":
        from .registry import FAMILIES
        for name, fam in FAMILIES.items():
            print(f"{name}: {', '.join(fam.dtypes)}")
        return 0
    print(__doc__.strip(), file=sys.stderr)
    return 2


if __name__ == "__main__":
    sys.exit(main())
