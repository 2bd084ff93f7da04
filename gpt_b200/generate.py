"""Command line of generation:  python -m gpt_b200.generate --model DIR --prompt 5,17,3 [--prompt ...] --max-new-tokens 16

Prompts and outputs are token ids; one line of output per prompt.  Without --prompt, prompts are read from standard input, one
per line.
"""
from __future__ import annotations

import argparse
import sys

from . import serving


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m gpt_b200.generate", description="Generate token ids with a model folder (config.json + weights).")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--prompt", action="append", help="token ids separated by commas or spaces; may be given several times")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--temperature", type=float, default=0.0, help="0: the most likely token")
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--max-sequences", type=int, default=8, help="sequences served at the same time")
    ap.add_argument("--step-tokens", type=int, default=2048, help="most tokens per step")
    a = ap.parse_args(argv)
    lines = a.prompt if a.prompt else [line for line in sys.stdin if line.strip()]
    prompts = [[int(t) for t in line.replace(",", " ").split()] for line in lines]
    model = serving.load_model(a.model, a.dtype)
    try:
        for out in serving.generate(model, prompts, a.max_new_tokens, a.temperature, a.seed, max_sequences=a.max_sequences, step_tokens=a.step_tokens):
            print(" ".join(str(t) for t in out))
    finally:
        model.close_model()
    return 0


if __name__ == "__main__":
    sys.exit(main())
