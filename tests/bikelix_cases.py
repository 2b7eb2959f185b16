"""Small configurations of the Bikelix decoder and helpers shared by its tests."""
import torch

import bikelix_oracle as oracle
from chunk_attn.models.bikelix import BikelixConfig, BikelixForCausalLM
from chunk_attn.models.bikelix.modeling_bikelix import random_weights
from gagorax_cases import Driver, error, tokens_for  # noqa: F401


def latent(heads, dim, rot, vdim, q_rank, kv_rank, window, scale=None, base=10000.0, kv_from=None, ff=None, limit=2.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "mask": {"size": window},
         "scale": (dim + rot) ** -0.5 if scale is None else scale, "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(width, vocab, layers, eps=1e-5, alpha=1.5, embed_scale=0.7, softcap=20.0):
    return {"architecture": "Bikelix", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}, "postln_alpha": alpha, "logit_softcap": softcap}


CONFIGS = {
    # nothing is a multiple of anything convenient; readers of two layers, with other heads, value sizes, scales and windows
    "odd": config(100, 131, [latent(3, 20, 12, 28, 36, 44, 37, base=500.0, ff=52), latent(5, 12, 6, 20, 28, 50, 90, scale=0.4),
                             latent(7, 36, 12, 12, 44, 44, 150, scale=0.1, base=500.0, kv_from=0, ff=76, limit=0.8),
                             latent(2, 28, 6, 44, 20, 50, 11, kv_from=1)], eps=1e-4, alpha=2.2, embed_scale=1.3, softcap=9.0),
    # whole lines in the cache, windows of whole chunks, many heads
    "wide": config(128, 200, [latent(16, 64, 64, 64, 96, 192, 128, ff=256), latent(16, 64, 64, 64, 96, 192, 128, kv_from=0),
                              latent(40, 32, 64, 32, 64, 192, 64, kv_from=0, ff=64, limit=1.0)], eps=1e-6, alpha=1.0),
    # sizes of large models' heads, one head per token row group, latents of 512
    "large": config(192, 96, [latent(4, 128, 64, 128, 160, 512, 200, ff=128), latent(2, 128, 64, 128, 96, 512, 1, kv_from=0),
                              latent(4, 128, 64, 128, 160, 512, 200)]),
    # more query rows than a block holds
    "heads": config(64, 70, [latent(72, 8, 8, 8, 16, 24, 70, ff=32)]),
}


def make(cfg, dtype, seed=0, weights=None, **engine):
    c = BikelixConfig.from_dict(cfg, torch_dtype=dtype, torch_device="cuda:0", **engine)
    w = random_weights(c, seed) if weights is None else weights
    return BikelixForCausalLM(c, w), {k: v.double().numpy() for k, v in w.items()}


TOL = {torch.float32: 3e-5, torch.bfloat16: 0.03}


def reference(cfg, weights, tokens):
    return oracle.forward(tokens, weights, cfg)[0]
