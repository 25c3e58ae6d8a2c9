"""Command line: sample token ids from any model the registry knows.

    python -m lighterpp_b200 generate --model PATH --prompt 1,2,3 -n 32 [--temperature T] [--penalty P] [--seed S]
                                      [--dtype bfloat16|float32] [--context N]

PATH is a GGUF or llama2.c file or a model folder (config.json + model.safetensors).  Prints the sampled ids.
"""
from __future__ import annotations

import argparse
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="lighterpp_b200", description="B200 decode engine")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="sample token ids after a prompt of token ids")
    g.add_argument("--model", required=True)
    g.add_argument("--prompt", required=True, help="token ids with commas between them")
    g.add_argument("-n", type=int, default=32, help="tokens to sample")
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--penalty", type=float, default=1.0)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--dtype", default="", choices=["", "bfloat16", "float32"], help="precision of a model folder")
    g.add_argument("--context", type=int, default=0, help="cache positions of a model folder")
    a = ap.parse_args(argv)
    from .build import ensure_built
    ensure_built()
    from .models import load_engine
    from .session import Session
    prompt = [int(t) for t in a.prompt.split(",")]
    eng = load_engine(a.model, a.dtype, a.context or len(prompt) + a.n)
    try:
        out = Session(eng).generate(prompt, a.n, a.temperature, a.penalty, a.seed)
    finally:
        eng.close()
    print(",".join(str(t) for t in out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
