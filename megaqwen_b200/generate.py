"""Greedy generation from the command line, for any registered model.

    python -m megaqwen_b200.generate MODEL_DIR --ids 5,17,3 --max-new 16
    python -m megaqwen_b200.generate MODEL_DIR --prompt "..."       # needs a tokenizer beside the weights
    python -m megaqwen_b200.generate --list

Prints the generated token ids (with --prompt the text), as they come.
"""
from __future__ import annotations

import argparse
import sys

from .registry import MODELS


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="megaqwen_b200.generate", description="greedy generation with a registered model")
    ap.add_argument("model", nargs="?", help="model directory (config.json and safetensors)")
    ap.add_argument("--list", action="store_true", help="list the registered models and exit")
    ap.add_argument("--ids", help="prompt as token ids with commas between them")
    ap.add_argument("--prompt", help="prompt as text")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--max-seq-len", type=int, default=2048)
    ap.add_argument("--stop", default="", help="token ids that end the generation, with commas between them")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    args = ap.parse_args(argv)
    if args.list:
        for entry in MODELS.values():
            print(f"{entry.name}: {', '.join(entry.dtypes)}")
        return 0
    if not args.model or (args.ids is None) == (args.prompt is None):
        ap.error("a model directory and one of --ids and --prompt are needed")

    from .csrc.build import build
    from .generators import MegakernelPrefillGenerator
    from .registry import find_model
    build(name=find_model(args.model).library)
    gen = MegakernelPrefillGenerator(args.model, args.max_seq_len, args.max_seq_len, dtype=args.dtype)
    if args.prompt is not None:
        if gen.tokenizer is None:
            sys.stderr.write("no tokenizer beside the weights: give the prompt as --ids\n")
            return 2
        for piece in gen.generate_stream(args.prompt, args.max_new):
            print(piece, end="", flush=True)
        print()
        return 0
    stops = [int(t) for t in args.stop.split(",") if t]
    print(" ".join(str(t) for t in gen.generate_ids([int(t) for t in args.ids.split(",")], args.max_new, stops)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
