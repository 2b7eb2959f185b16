"""Greedy generation from the command line, through the continuous-batching host.

    python -m chunk_attn.generate --model DIR --max-new-tokens 32 < prompts

Each line of standard input is one prompt, token ids separated by blanks; the completed token ids of each prompt are
printed in the order of the prompts.  All prompts are served together, up to --max-batch-size at a time.
"""
import argparse
import sys

import torch

from .models.model_host import ModelHost
from .models.registry import load_model


def main(argv=None):
    ap = argparse.ArgumentParser(prog="chunk_attn.generate", description="Greedy generation from token ids on standard input.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default=None, choices=["bfloat16", "float16", "float32"])
    ap.add_argument("--device", default="cuda:0")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--max-batch-size", type=int, default=32)
    a = ap.parse_args(argv)
    prompts = [[int(t) for t in line.split()] for line in sys.stdin if line.strip()]
    model = load_model(a.model, dtype=getattr(torch, a.dtype) if a.dtype else None, device=a.device)
    with ModelHost(model, model.create_kv_caches(), max_batch_size=a.max_batch_size) as host:
        pending = []
        for p in prompts:
            pending.append(host.predict_async(p, a.max_new_tokens))
        for seq in pending:
            print(" ".join(str(t) for t in seq.get_result()))
    return 0


if __name__ == "__main__":
    sys.exit(main())
