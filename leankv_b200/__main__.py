"""Command line: ``python -m leankv_b200 {generate,trace,architectures}``."""

from __future__ import annotations

import argparse
import json
import sys


def main(argv=None) -> int:
    argv = list(sys.argv[1:] if argv is None else argv)
    if argv[:1] == ["trace"]:
        from .trace import main as trace_main

        return trace_main(argv[1:])
    ap = argparse.ArgumentParser(prog="python -m leankv_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    sub.add_parser("trace", help="replay token portions and write logits (see `trace --help`)")
    sub.add_parser("architectures", help="list the architectures the registry knows")
    g = sub.add_parser("generate", help="greedy generation from a model folder")
    g.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    g.add_argument("--prompt", required=True, help="prompt token ids, separated by commas")
    g.add_argument("--max-new-tokens", type=int, default=32)
    g.add_argument("--dtype", default=None, help="storage type (default: the architecture's)")
    g.add_argument("--max-seq-len", type=int, default=None)
    g.add_argument("--device", default="cuda:0")
    args = ap.parse_args(argv)

    from . import registry

    if args.command == "architectures":
        print("\n".join(registry.architectures()))
        return 0
    prompt = [int(t) for t in args.prompt.split(",")]
    limit = args.max_seq_len or len(prompt) + args.max_new_tokens + 1
    engine = registry.load_engine(args.model, args.device, args.dtype, max_seq_len=limit)
    print(json.dumps({"tokens": engine.generate(prompt, args.max_new_tokens)}))
    return 0


if __name__ == "__main__":
    sys.exit(main())
