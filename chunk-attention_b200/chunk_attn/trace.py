"""Feeds recorded token ids to a model and writes the logits it gives them, without sampling.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Every line of standard input is a JSON object, one step:

    {"step": 7, "entries": [{"id": "x", "tokens": [11, 4], "want": [1]}], "end": ["x"]}

An entry continues the request of that id (or starts it) by its tokens and asks for logits at the given indexes into them;
requests named in `end` leave the caches once the step has run.  Where anything is asked for, <out>/<step>.f32 receives
little-endian fp32 rows [asked, vocab], entry by entry; "done <step>" on standard output follows each step.

The work is the model's step function on its own caches: each entry is a span of the step.
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
        """entries: [(id, tokens, indexes to return)].  Returns fp32 logits [n, vocab] on the CPU, or None."""
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
    ap.add_argument("--max-tokens", type=int, required=True, help="upper bound of the tokens alive at once: sizes the KV pools")
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
