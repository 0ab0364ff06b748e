"""Replays a recorded request trace through a decoder and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

An entry carries the next tokens of a request; a request begins with its first
entry and keeps its cache and state until an ``end`` list names it.  The
decoder holds one sequence, so a step has one entry and a request begins when
the one before has ended.  For a step in which places are wanted, ``--out``
receives ``<step>.f32``: their logits as little-endian 32-bit floats, [wanted,
vocab].  After every step a line ``done <step>`` follows on standard output.

The tokens are given, nothing is sampled; the decoder is the one generation
uses (``registry.build_decoder``), one token at a time through its decode step
and more through its prefill.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

EXIT_DTYPE = 3


class TraceRunner:
    def __init__(self, decoder, out_dir: str):
        self.decoder = decoder
        self.out_dir = out_dir
        self.live = None

    def run_step(self, step: dict) -> None:
        entries = step["entries"]
        if len(entries) > 1:
            raise ValueError("a step has one entry: the decoder holds one sequence")
        for entry in entries:
            if self.live is None:
                self.decoder.reset()
                self.live = entry["id"]
            elif self.live != entry["id"]:
                raise ValueError(f"request {entry['id']!r} begins before {self.live!r} has ended")
            logits = self.decoder.step_logits(entry["tokens"], entry["want"])
            if entry["want"]:
                path = os.path.join(self.out_dir, f"{step['step']}.f32")
                with open(path, "wb") as fh:
                    fh.write(logits.float().cpu().contiguous().numpy().astype("<f4").tobytes())
        for name in step.get("end", []):
            if name == self.live:
                self.decoder.reset()
                self.live = None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a request trace and write logits")
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens a live request holds")
    ap.add_argument("--max-prefill", type=int, default=2048, help="most tokens of one prefill launch")
    args = ap.parse_args(argv)

    from .registry import find_model
    entry = find_model(args.model)
    if args.dtype not in entry.dtypes:
        sys.stderr.write(f"{entry.name} does not run in {args.dtype}\n")
        return EXIT_DTYPE
    from .csrc.build import build
    build(name=entry.library)
    from .registry import build_decoder
    decoder, _ = build_decoder(args.model, args.max_tokens + 1, min(args.max_prefill, args.max_tokens + 1), dtype=args.dtype)
    runner = TraceRunner(decoder, args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        runner.run_step(step)
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
