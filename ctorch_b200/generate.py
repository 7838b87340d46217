"""Command line of the generation loop: token ids in, token ids out.

    python -m ctorch_b200.generate --model DIR [--dtype bf16|f32] [--steps N] [--temperature T] [--seed S] PROMPT...

DIR holds config.json and model.safetensors; the design is chosen by the configuration.  Every PROMPT is a comma-separated list
of token ids; prompts of unequal length run as one batch.  Prints one line of generated ids per prompt.
"""
from __future__ import annotations

import argparse
import sys


def main(argv: list[str] | None = None) -> int:
    parser = argparse.ArgumentParser(prog="ctorch_b200.generate", description=__doc__.split("\n")[0])
    parser.add_argument("--model", required=True)
    parser.add_argument("--dtype", default="bf16", choices=["bf16", "f32"])
    parser.add_argument("--steps", type=int, default=16)
    parser.add_argument("--temperature", type=float, default=None, help="sample at this temperature instead of the greedy choice")
    parser.add_argument("--seed", type=int, default=0)
    parser.add_argument("prompts", nargs="+", metavar="PROMPT")
    args = parser.parse_args(argv)
    import ctorch_b200 as B
    model = B.LanguageModel.load(args.model, dtype=args.dtype)
    prompts = [[int(t) for t in p.split(",")] for p in args.prompts]
    for row in model.generate(prompts, args.steps, temperature=args.temperature, seed=args.seed):
        print(",".join(str(int(t)) for t in row))
    return 0


if __name__ == "__main__":
    sys.exit(main())
