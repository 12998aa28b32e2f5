"""Replays a trace of token steps through a model: given tokens in, logits out, nothing sampled.

Steps come on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every request lives in a sequence slot of the model.  An entry's tokens continue its sequence: a single token of a running
sequence is a decode step (all such entries of a step share one batched pass over the weights), anything else is a prompt
portion.  `want` lists the places among the tokens whose logits are written to OUT/<step>.f32 (little-endian f32
[wanted, vocab], in entry order); `end` lists requests whose slots are given back after the step.  After each step a line
"done <step>" is printed.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


class TraceRunner:
    """Drives the slots of a loaded model step by step."""

    def __init__(self, model):
        self.model = model
        self.slots = {}   # request id -> (slot, length)

    def step(self, entries, end=()):
        """Logits [wanted, vocab] of a step's entries, in order."""
        out = [None] * len(entries)
        single = []
        for i, e in enumerate(entries):
            rid, toks, want = e["id"], e["tokens"], e.get("want", [])
            if rid not in self.slots:
                self.slots[rid] = [self.model.seq_create(), 0]
            slot, length = self.slots[rid]
            if len(toks) == 1 and length > 0:
                single.append((i, slot, toks[0], want))
            elif toks:
                out[i] = self.model.seq_prefill_logits(slot, toks, length, want)
            self.slots[rid][1] += len(toks)
        if single:
            rows = self.model.decode_batch_logits([t for _, _, t, _ in single], [s for _, s, _, _ in single])
            for r, (i, _, _, want) in enumerate(single):
                out[i] = np.repeat(rows[r:r + 1], len(want), axis=0)
        for rid in end:
            if rid in self.slots:
                self.model.seq_destroy(self.slots.pop(rid)[0])
        wanted = [o for o in out if o is not None and len(o)]
        return np.concatenate(wanted) if wanted else np.empty((0, self.model.config().vocab_size), np.float32)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="model folder (config.json, model.safetensors) or GGUF file")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32", "default"], help="arithmetic of a model folder")
    ap.add_argument("--out", required=True, help="folder for the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", type=int, default=0)
    args = ap.parse_args(argv)
    from . import build
    build.build()
    from .model import load_model_cuda
    model = load_model_cuda(args.model, max(1, args.max_tokens), args.device, args.dtype)
    runner = TraceRunner(model)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = runner.step(s.get("entries", []), s.get("end", []))
        if len(logits):
            tmp = os.path.join(args.out, f".{s['step']}.part")
            logits.astype("<f4").tofile(tmp)
            os.replace(tmp, os.path.join(args.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    model.close()
    return 0
