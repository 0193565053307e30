"""Command line.

    python -m torchburn_b200 generate --model DIR --tokens 1,2,3 --max-new 32 [--dtype ...] [sampling options]
    python -m torchburn_b200 designs
"""
from __future__ import annotations

import argparse
import sys

from . import models
from .speculative import BatchedDecoder


def _generate(a) -> int:
    prompts = [[int(t) for t in p.split(",")] for p in a.tokens]
    if len(prompts) == 1 or a.max_batch == 1:
        dec = models.load_model(a.model, a.dtype, a.max_seq_len, build=True)
        dec.seed(a.seed)
        for p in prompts:
            dec.reset_kv_cache()
            if len(p) > 1:
                dec.prefill_tokens(p[:-1], 0)
            # generate_loop emits its first token as it is: the last prompt token, dropped here
            toks, _ = dec.generate_loop(p[-1], len(p) - 1, a.max_new + 1, a.temperature, a.top_k, a.repetition_penalty, a.top_p,
                                        a.eos, recent_seed=p[:-1])
            print(",".join(map(str, toks[1:])))
        return 0
    dec = models.load_model(a.model, a.dtype, a.max_seq_len, build=True, max_batch=a.max_batch)
    batched = BatchedDecoder(lambda: dec, a.max_batch, a.temperature, a.top_k, a.eos)
    for toks in batched.generate_batch(prompts, a.max_new):
        print(",".join(map(str, toks)))
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="torchburn_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="continue prompts of token ids")
    g.add_argument("--model", required=True)
    g.add_argument("--tokens", required=True, action="append", help="comma-separated ids; once per prompt")
    g.add_argument("--max-new", type=int, default=32)
    g.add_argument("--dtype", default=None)
    g.add_argument("--max-seq-len", type=int, default=None)
    g.add_argument("--max-batch", type=int, default=1)
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=40)
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--repetition-penalty", type=float, default=1.0)
    g.add_argument("--eos", type=int, default=None)
    g.add_argument("--seed", type=int, default=1)
    sub.add_parser("designs", help="the registered model designs")
    a = ap.parse_args(argv)
    if a.cmd == "designs":
        print("\n".join(models.designs()))
        return 0
    return _generate(a)


if __name__ == "__main__":
    sys.exit(main())
