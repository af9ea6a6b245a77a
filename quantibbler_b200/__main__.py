"""Command line: greedy generation from token ids with any model the registry knows.

    python -m quantibbler_b200 generate --model DIR --prompt 5,17,3 --max-tokens 32
    python -m quantibbler_b200 trace --model DIR --out OUT < steps.jsonl

Prints one JSON object (token ids in and out: text needs the model's tokenizer, which is not part
of this package)."""

from __future__ import annotations

import argparse
import json
import sys


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else argv
    if argv[:1] == ["trace"]:
        from .trace import main as trace_main
        return trace_main(argv[1:])
    ap = argparse.ArgumentParser(prog="quantibbler_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy continuation of a prompt")
    g.add_argument("--model", required=True, help="a folder with config.json, a model directory or a blob")
    g.add_argument("--prompt", required=True, help="token ids, with commas between them")
    g.add_argument("--max-tokens", type=int, default=32)
    g.add_argument("--eos", type=int, default=None, help="token id that ends the generation")
    g.add_argument("--dtype", choices=("bfloat16", "float32"), default=None, help="default: the model's own")
    sub.add_parser("trace", help="replay a trace of token ids (see bin/trace_run)")
    a = ap.parse_args(argv)
    from .gpu import GpuContext
    from .registry import load_decoder
    prompt = [int(t) for t in a.prompt.split(",")]
    settings = {} if a.dtype is None else {"serving": a.dtype}
    decoder = load_decoder(GpuContext.init(), a.model, max_seq=len(prompt) + max(a.max_tokens, 1), **settings)
    print(json.dumps(decoder.generate(prompt, a.max_tokens, a.eos)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
