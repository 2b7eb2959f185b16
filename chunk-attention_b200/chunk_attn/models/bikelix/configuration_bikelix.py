"""Configuration of the Bikelix decoder: the model's own fields as config.json names them, and the engine's."""
import dataclasses
import json

import torch

MIXERS = {"latent_attention": ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot", "mask")}
FEED_FORWARDS = {"dense": ("ff", "limit")}


def _require(spec, names, where):
    missing = [k for k in names if k not in spec]
    if missing:
        raise ValueError("%s: fields missing: %s" % (where, ", ".join(missing)))


@dataclasses.dataclass
class BikelixConfig:
    vocab: int
    width: int
    layers: list
    norm: dict
    embedding: dict
    postln_alpha: float
    logit_softcap: float
    # engine side
    chunk_size: int = 64
    kvcache_gb: float = 0.0       # 0: size the pools from the device's free memory
    prefill_portion: int = 8192   # tokens of prompts run through the layers at a time
    state_slots: int = 16         # grows on demand
    torch_dtype: torch.dtype = torch.bfloat16
    torch_device: str = "cuda:0"

    def __post_init__(self):
        if self.torch_dtype not in (torch.bfloat16, torch.float32):
            raise NotImplementedError("Bikelix runs in bfloat16 or float32")
        if self.prefill_portion < 1:
            raise ValueError("prefill_portion must be positive")
        if not self.logit_softcap > 0:
            raise ValueError("logit_softcap must be positive")
        _require(self.norm, ("eps",), "norm")
        _require(self.embedding, ("scale",), "embedding")
        for i, layer in enumerate(self.layers):
            kind, m, mlp = layer["type"], layer["mixer"], layer.get("mlp")
            if kind not in MIXERS:
                raise NotImplementedError("layer %d: unknown mixer %r" % (i, kind))
            _require(m, MIXERS[kind], "layer %d: mixer" % i)
            if m["rot_dim"] % 2 or m["rot"]["dims"] != m["rot_dim"]:
                raise ValueError("layer %d: the rotated part is rotated as a whole, and has an even size" % i)
            if m["mask"]["size"] < 1:
                raise ValueError("layer %d: a window holds at least the position itself" % i)
            if m["kv_rank"] > 1024 or m["kv_rank"] + m["rot_dim"] > 1152:
                raise NotImplementedError("layer %d: latents of up to 1024 elements, rows of up to 1152" % i)
            owner = m.get("kv_from")
            if owner is not None:
                if not 0 <= owner < i:
                    raise ValueError("layer %d: kv_from must name an earlier layer" % i)
                o = self.layers[owner]["mixer"]
                if o.get("kv_from") is not None:
                    raise ValueError("layer %d: kv_from must name a layer with a latent of its own" % i)
                if any(o[k] != m[k] for k in ("kv_rank", "rot_dim", "rot")):
                    raise ValueError("layer %d: latent and rotation must be those of layer %d" % (i, owner))
            if mlp is not None:
                if mlp["kind"] not in FEED_FORWARDS:
                    raise NotImplementedError("layer %d: unknown feed-forward %r" % (i, mlp["kind"]))
                _require(mlp, FEED_FORWARDS[mlp["kind"]], "layer %d: feed-forward" % i)

    @property
    def eps(self):
        return float(self.norm["eps"])

    @classmethod
    def from_dict(cls, d, **engine):
        names = {f.name for f in dataclasses.fields(cls)}
        d = {k: v for k, v in d.items() if k in names}
        d.update(engine)
        if isinstance(d.get("torch_dtype"), str):
            d["torch_dtype"] = getattr(torch, d["torch_dtype"])
        return cls(**d)

    @classmethod
    def from_json_file(cls, path, **engine):
        with open(path) as f:
            return cls.from_dict(json.load(f), **engine)
