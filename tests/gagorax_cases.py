"""Small configurations of the Gagorax decoder and helpers shared by its tests."""
import numpy as np
import torch

import gagorax_oracle as oracle
from chunk_attn.models.gagorax import GagoraxConfig, GagoraxForCausalLM
from chunk_attn.models.gagorax.modeling_gagorax import random_weights


def attention(heads, kv, dim, vdim, rot, scale=None, base=10000.0, ff=None):
    return {"type": "attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
                      "scale": dim ** -0.5 if scale is None else scale}}


def mamba(inner, state, rank, conv, ff=None):
    return {"type": "mamba1", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"inner": inner, "state": state, "dt_rank": rank, "conv": conv}}


def lightning(dim, vdim, decay, ff=None):
    return {"type": "lightning", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": decay}}


def config(width, vocab, layers, eps=1e-5, logit_scale=1.0):
    return {"architecture": "Gagorax", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}, "logit_scale": logit_scale}


CONFIGS = {
    # nothing is a multiple of anything convenient; every layer type with and without a feed-forward
    "odd": config(100, 131, [attention(6, 2, 40, 24, 24, scale=0.3, base=500.0, ff=164), mamba(112, 5, 7, 4),
                             lightning(24, 40, [0.5, 0.9, 0.99], ff=72), mamba(130, 40, 3, 2, ff=64), attention(3, 3, 20, 36, 8),
                             lightning(36, 20, [0.97])], eps=1e-4, logit_scale=0.7),
    # head sizes of large models, one key/value head per query head
    "wide": config(128, 200, [attention(2, 2, 128, 128, 128, ff=256), mamba(256, 16, 8, 1), lightning(128, 128, [0.95, 1.0])],
                   eps=1e-6, logit_scale=1.5),
    # many query heads on one key/value head; 64-element heads; recurrent layers first and last
    "grouped": config(192, 96, [lightning(64, 64, [0.8, 0.999]), attention(16, 1, 64, 64, 32, base=1e6), mamba(192, 16, 12, 4),
                                attention(8, 4, 128, 64, 64, ff=128), mamba(64, 8, 4, 3)]),
    "recurrent": config(64, 70, [mamba(96, 16, 6, 4), lightning(16, 16, [0.9, 0.7])]),  # no attention layer at all
}


def make(cfg, dtype, seed=0, weights=None, **engine):
    c = GagoraxConfig.from_dict(cfg, torch_dtype=dtype, torch_device="cuda:0", **engine)
    w = random_weights(c, seed) if weights is None else weights
    return GagoraxForCausalLM(c, w), {k: v.double().numpy() for k, v in w.items()}


def tokens_for(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def error(got, want):
    """Worst over the rows: rms difference without its mean over the vocabulary, in units of the logits' spread."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return float(np.sqrt((d ** 2).mean(-1)).max() / want.std())


TOL = {torch.float32: 3e-5, torch.bfloat16: 0.1}


class Driver:
    """Feeds requests to a model's step function by name and collects the logits of every position."""

    def __init__(self, model, max_tokens=4096):
        self.model, self.caches, self.order, self.got = model, model.create_kv_caches(max_tokens=max_tokens), [], {}

    def step(self, entries):
        rows = [self.order.index(n) if n in self.order else None for n, _ in entries]
        x, spans, out = self.model.step(rows, [t for _, t in entries], self.caches)
        for (n, _), was, r in zip(entries, rows, out):
            if was is None:
                self.order.insert(r, n)
        lg = self.model.head_logits(x, torch.arange(x.shape[0], dtype=torch.int32, device=x.device)).cpu().numpy()
        base = 0
        for n, t in entries:
            self.got.setdefault(n, []).append(lg[base:base + len(t)])
            base += len(t)

    def end(self, name):
        row = self.order.index(name)
        for c in self.caches:
            c.remove_seq(row)
        del self.order[row]

    def logits(self, name):
        return np.concatenate(self.got[name])

    def clean(self):
        return all(c.device_status() == 0 for c in self.caches[:-1])


def reference(cfg, weights, tokens):
    return oracle.forward(tokens, weights, cfg)[0]
