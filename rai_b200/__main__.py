"""Command line over a checkpoint folder (config.json and *.safetensors), for every architecture the library has.

    python -m rai_b200 generate --model DIR --prompt 11,8,402 [--prompt ...] --steps 32
    python -m rai_b200 trace --model DIR --out DIR --max-tokens N < steps.jsonl       (also: bin/trace_run)

`generate` takes token ids (the library has no tokenizer) and prints the generated ids of each prompt on a line.
"""
from __future__ import annotations

import argparse
import sys


def generate(argv) -> int:
    ap = argparse.ArgumentParser(prog="rai_b200 generate")
    ap.add_argument("--model", required=True, help="checkpoint folder")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; repeat for a batch")
    ap.add_argument("--steps", type=int, default=32, help="tokens to generate per prompt")
    ap.add_argument("--repeat-penalty", type=float, default=0.0, help="below 1: none")
    ap.add_argument("--repeat-last-n", type=int, default=64)
    ap.add_argument("--eos", type=int, default=-1, help="end-of-sequence token id")
    a = ap.parse_args(argv)
    prompts = [[int(t) for t in p.split(",")] for p in a.prompt]

    from . import _lib, build
    if not build.LIB.exists():
        build.build()
    from .device import Cuda
    from .models import Model
    longest = max(len(p) for p in prompts)
    m = Model.from_pretrained(a.model, _lib.BF16 if a.dtype == "bfloat16" else _lib.F32, Cuda(0), len(prompts),
                              longest + a.steps, len(prompts) * longest)
    if a.repeat_penalty >= 1.0 or a.eos >= 0:
        m.set_sampling(a.repeat_penalty, a.repeat_last_n, a.eos)
    for row in m.generate_ragged(prompts, a.steps):
        out = row.tolist()
        if a.eos in out:
            out = out[:out.index(a.eos) + 1]
        print(",".join(str(t) for t in out))
    m.close()
    return 0


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else argv
    if argv[:1] == ["generate"]:
        return generate(argv[1:])
    if argv[:1] == ["trace"]:
        from .trace import main as trace
        return trace(argv[1:])
    print(__doc__.strip())
    return 0 if argv[:1] in (["-h"], ["--help"]) else 2


if __name__ == "__main__":
    sys.exit(main())
