"""Replays a trace through a model: token ids come in step by step, logits go out.  Nothing is sampled.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps are read from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

`entries` are the next tokens of each request and the places among them whose logits are wanted; `end` names the
requests that are finished after the step.  A step that wants something writes <out>/<step>.f32, the logits in the order
of the entries, as little-endian fp32; after every step the line "done <step>" is printed.

It drives the model's own step function and caches: each entry is a span of the step, continued from what earlier steps
left.
"""
import argparse
import json
import os
import sys

import torch

from .models.registry import load_model


class TraceRunner:
    def __init__(self, model, max_tokens):
        self.model = model
        self.caches = model.create_kv_caches(max_tokens=max_tokens)
        self.order = []  # request ids in the caches' row order

    def step(self, entries, end):
        """entries: [(id, tokens, wanted places)].  Returns the wanted logits, fp32 [n, vocab] on the CPU, or None."""
        logits = None
        if entries:
            rows = [self.order.index(i) if i in self.order else None for i, _, _ in entries]
            x, spans, got = self.model.step(rows, [t for _, t, _ in entries], self.caches)
            for (i, _, _), was, r in zip(entries, rows, got):
                if was is None:
                    self.order.insert(r, i)
            want, base = [], 0
            for _, tokens, places in entries:
                want += [base + p for p in places]
                base += len(tokens)
            if want:
                idx = torch.tensor(want, dtype=torch.int32, device=x.device)
                logits = self.model.head_logits(x, idx).cpu()
        for i in end:
            row = self.order.index(i)
            for cache in self.caches:
                cache.remove_seq(row)
            del self.order[row]
        return logits


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replays a trace of token ids through a model and writes logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    a = ap.parse_args(argv)
    runner = TraceRunner(load_model(a.model, dtype=getattr(torch, a.dtype)), a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = runner.step([(e["id"], e["tokens"], e.get("want", [])) for e in s["entries"] if e["tokens"]], s.get("end", []))
        if logits is not None:
            path = os.path.join(a.out, "%d.f32" % s["step"])
            logits.numpy().astype("<f4").tofile(path + ".part")
            os.replace(path + ".part", path)
        print("done %d" % s["step"], flush=True)
    return 0
