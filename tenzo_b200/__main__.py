"""Command line of the runtime.

    python -m tenzo_b200 generate --model DIR --tokens 5,17,3 --n 32 [--dtype float32] [--temperature 0.7 --top-p 0.9 --top-k 40 --penalty 1.15]
    python -m tenzo_b200 trace ...        as bin/trace_run
    python -m tenzo_b200 models           architectures this library serves

A model is a folder whose config.json names its architecture. Prompts and results are token ids; decoding is greedy
unless a temperature is given.
"""
from __future__ import annotations

import argparse
import sys


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else list(argv)
    if argv[:1] == ["trace"]:
        from .trace import main as trace_main
        return trace_main(argv[1:])
    ap = argparse.ArgumentParser(prog="tenzo_b200", description="Serve a model folder on the GPU.")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="continue a prompt of token ids")
    g.add_argument("--model", required=True)
    g.add_argument("--tokens", required=True, help="prompt token ids, separated by commas or blanks")
    g.add_argument("--n", type=int, default=32, help="tokens to generate")
    g.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-p", type=float, default=0.9)
    g.add_argument("--top-k", type=int, default=40)
    g.add_argument("--penalty", type=float, default=1.0)
    sub.add_parser("models", help="list the architectures")
    sub.add_parser("trace", help="replay a token trace (bin/trace_run)")
    a = ap.parse_args(argv)
    if a.command == "models":
        from . import load_library
        lib, i = load_library(), 0
        while (name := lib.tenzo_ext_architecture(i)) is not None:
            print(name.decode())
            i += 1
        return 0
    from . import abi
    from .engine import Engine
    prompt = [int(t) for t in a.tokens.replace(",", " ").split()]
    with Engine.open(a.model, compute=a.dtype) as e:
        print(" ".join(map(str, e.generate(prompt, a.n, abi.TenzoSampling(a.temperature, a.top_p, a.top_k, a.penalty)))))
    return 0


if __name__ == "__main__":
    sys.exit(main())
