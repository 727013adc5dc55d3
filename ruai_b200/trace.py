"""Replays a trace: feeds given token ids through a model step by step and writes the logits that are asked for.

    trace_run --model DIR [--dtype bfloat16|float32] --out DIR [--max-tokens N]

Steps come on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

An entry brings a request's next tokens and the places among them whose logits are wanted; they continue from what
earlier steps left in the model's cache and states.  `end` names requests that are finished after the step.  The logits
go to OUT/<step>.f32 (little-endian f32, [wanted, vocab]); `done <step>` is printed after every step.  One request is
live at a time.
"""
import argparse
import json
import os
import sys

import numpy as np

from . import nn, registry


class Replay:
    """Steps of one live request over a model's `forward_rows`."""

    def __init__(self, model):
        self.model, self.live = model, None

    def step(self, entries, end):
        if len(entries) > 1:
            raise ValueError("one request per step")
        out = np.empty((0, self.model.vocab), np.float32)
        for e in entries:
            if self.live is None:
                self.model.cache_clear()
                self.live = e["id"]
            if e["id"] != self.live:
                raise ValueError(f"request {e['id']!r} began before {self.live!r} ended")
            if e["tokens"]:
                out = self.model.forward_rows(np.array([e["tokens"]], np.int32), e.get("want") or [])
        if self.live in end:
            self.model.cache_clear()
            self.live = None
        return out


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Feed token ids through a model step by step and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=registry.DTYPES)
    ap.add_argument("--bits", type=int, choices=(4, 8), help="quantize on loading (Llama, GPT-2)")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens a live request holds: sizes the cache ahead")
    a = ap.parse_args(argv)
    model = registry.load(nn.Device.cuda(0), a.model, a.dtype, a.bits)
    if a.max_tokens > 0:
        model.cache_reserve(1, min(a.max_tokens, model.max_positions))
    replay = Replay(model)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s.get("entries", []), s.get("end", []))
        if logits.shape[0]:
            logits.astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    return 0
