"""Greedy generation from the command line:

    python -m nn_b200.generate --model PATH --prompt 11,4,90 --new 32 [--dtype bfloat16|float32] [--max-seq N]

PATH is a model folder (config.json + model.safetensors) or a GGUF file; prompt and output are token ids.
"""
from __future__ import annotations

import argparse
import sys

from . import models
from .trace import DTYPES


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m nn_b200.generate", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompt", required=True, help="token ids with commas between them")
    ap.add_argument("--new", type=int, default=16, help="tokens to generate")
    ap.add_argument("--dtype", default="bfloat16", choices=sorted(DTYPES))
    ap.add_argument("--max-seq", type=int, default=0, help="positions held (default: prompt + new)")
    a = ap.parse_args(argv)
    prompt = [int(t) for t in a.prompt.split(",")]
    dec = models.load_model(a.model, max_seq=a.max_seq or len(prompt) + a.new, act_dtype=DTYPES[a.dtype])
    print(",".join(str(t) for t in dec.complete(prompt, a.new)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
