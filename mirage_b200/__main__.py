"""Command line: generation from a checkpoint directory on token ids.

    python -m mirage_b200 generate --model DIR --prompt 5,17,3 [--prompt ...] --max-new-tokens 16

Prints one JSON list of ids (prompt + new tokens) per prompt.
"""
from __future__ import annotations

import argparse
import json
import sys


def generate(a) -> int:
    import torch
    from . import load_runner
    prompts = [[int(t) for t in p.split(",")] for p in a.prompt]
    # the scheduler ends a request at the table's end, which every request must be able to reach
    seq = max(len(p) for p in prompts) + a.max_new_tokens
    slots = min(len(prompts), a.max_batch)
    pages = slots * -(-seq // a.page_size)
    runner = load_runner(a.model, getattr(torch, a.dtype), total_num_requests=len(prompts), max_seq_length=seq,
                         max_num_batched_requests=slots, max_num_batched_tokens=a.batch_tokens, max_num_pages=pages,
                         page_size=a.page_size, eos_token_id=a.eos, sampling_seed=a.sampling_seed)
    for ids in runner.generate(prompts, a.max_new_tokens):
        print(json.dumps(ids))
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m mirage_b200", description=__doc__,
                                 formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="generate from prompts given as token ids")
    g.add_argument("--model", required=True, help="checkpoint directory (config.json + *.safetensors)")
    g.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; may be repeated")
    g.add_argument("--max-new-tokens", type=int, default=16)
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    g.add_argument("--eos", type=int, default=-1)
    g.add_argument("--sampling-seed", type=int, default=None, help="Gumbel-max sampling instead of the greedy choice")
    g.add_argument("--max-batch", type=int, default=16, help="requests that run at the same time")
    g.add_argument("--batch-tokens", type=int, default=64, help="tokens of one launch")
    g.add_argument("--page-size", type=int, default=64)
    a = ap.parse_args(argv)
    return generate(a)


if __name__ == "__main__":
    sys.exit(main())
