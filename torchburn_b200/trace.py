"""Replays a trace of token ids through a model and writes logits (the program behind bin/trace_run).

Reads one JSON object a line from standard input,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}

feeds every entry's tokens to the decoder as the continuation of its request, writes the logits at the wanted
places to OUT/<step>.f32 (little-endian float32, in the order of entries and places) and answers
"done <step>".  Requests named in "end" give their sequence back after the step.  Exit code 3: the model's
design is not served in the asked dtype."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Tuple

import numpy as np

from . import _lib, models


class Requests:
    """Live requests on the decoder's sequences: id -> (sequence, next position)."""

    def __init__(self, decoder):
        self.decoder = decoder
        self.live: Dict[str, Tuple[int, int]] = {}
        self.free: List[int] = list(range(decoder.max_batch))

    def feed(self, rid: str, tokens, want) -> np.ndarray:
        if rid not in self.live:
            if not self.free:
                raise RuntimeError(f"request {rid!r}: all {self.decoder.max_batch} sequences are in use")
            self.live[rid] = (self.free.pop(0), 0)
        seq, at = self.live[rid]
        out = self.decoder.extend(tokens, at, want, seq)
        self.live[rid] = (seq, at + len(tokens))
        return out

    def end(self, rid: str) -> None:
        if rid in self.live:
            seq, _ = self.live.pop(rid)
            self.decoder.reset_sequence(seq)
            self.free.append(seq)


def run(decoder, lines, out_dir: str, answer) -> None:
    reqs = Requests(decoder)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = [reqs.feed(e["id"], e["tokens"], e["want"]) for e in step["entries"] if e["tokens"]]
        if _lib.lib().tb_device_fault_flag() != 0:
            raise RuntimeError("a bounded device-side wait ran out")
        if any(r.size for r in rows):
            np.concatenate(rows).astype("<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        for rid in step.get("end", ()):
            reqs.end(rid)
        answer(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replays a trace of token ids through a model and writes logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, help="bfloat16, float32 or whatever else the model's design is served in")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=None, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=1, help="most requests that are live at any time")
    a = ap.parse_args(argv)
    try:
        dec = models.load_model(a.model, a.dtype, max_seq_len=a.max_tokens, build=True, max_batch=a.max_requests)
    except NotImplementedError as e:
        print(e, file=sys.stderr)
        return 3
    os.makedirs(a.out, exist_ok=True)

    def answer(text):
        print(text, flush=True)

    run(dec, sys.stdin, a.out, answer)
    return 0


if __name__ == "__main__":
    sys.exit(main())
