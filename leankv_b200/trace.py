"""Replays a trace: token portions read from standard input go through a model's engine, step by step, and
the logits asked for are written to files. Nothing is sampled.

One JSON object a line: ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``. A step brings
the next tokens of one request; ``want`` lists places among them; ``end`` names the requests that are
finished. Logits go to ``OUT/<step>.f32`` (little-endian fp32 [wanted][vocab]); ``done <step>`` follows.
"""

from __future__ import annotations

import argparse
import json
import os
import sys

REFUSED = 3


def replay(engine, lines, out_dir: str, say) -> None:
    """The engine serves one sequence at a time: a request is live from its first tokens until its end."""
    live = None
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        if len(step["entries"]) > 1:
            raise ValueError("this engine serves one request at a time")
        for e in step["entries"]:
            if live is None:
                engine.reset()
                live = e["id"]
            elif live != e["id"]:
                raise ValueError(f"request {e['id']} begins before {live} has ended")
            logits = engine.extend(e["tokens"], e["want"])
            if e["want"]:
                data = logits.cpu().numpy().astype("<f4", copy=False)
                part = os.path.join(out_dir, f".{step['step']}.part")
                data.tofile(part)
                os.replace(part, os.path.join(out_dir, f"{step['step']}.f32"))
        for i in step["end"]:
            if i != live:
                raise ValueError(f"request {i} is not live")
            engine.reset()
            live = None
        say(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens a live request holds")
    args = ap.parse_args(argv)

    from . import registry
    from .checkpoint import read_config

    if not registry.supports(read_config(args.model), args.dtype):
        sys.stderr.write(f"this model does not run in {args.dtype}\n")
        return REFUSED
    import torch

    torch.set_float32_matmul_precision("highest")
    torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
    engine = registry.load_engine(args.model, "cuda:0", args.dtype, max_seq_len=args.max_tokens)

    def say(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    replay(engine, sys.stdin, args.out, say)
    return 0


if __name__ == "__main__":
    sys.exit(main())
