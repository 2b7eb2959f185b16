"""Configuration of the Gagorax decoder: the model's own fields as config.json names them, and the engine's."""
import dataclasses
import json

import torch

MIXERS = {
    "mamba1": ("inner", "state", "dt_rank", "conv"),
    "attention": ("heads", "kv_heads", "dim", "vdim", "scale", "rot"),
    "lightning": ("heads", "dim", "vdim", "decay"),
}


@dataclasses.dataclass
class GagoraxConfig:
    vocab: int
    width: int
    layers: list
    norm: dict
    logit_scale: float = 1.0
    # engine side
    chunk_size: int = 64
    kvcache_gb: float = 0.0       # 0: size the pools from the device's free memory
    prefill_portion: int = 8192   # tokens of prompts run through the layers at a time
    state_slots: int = 16         # grows on demand
    torch_dtype: torch.dtype = torch.bfloat16
    torch_device: str = "cuda:0"

    def __post_init__(self):
        if self.torch_dtype not in (torch.bfloat16, torch.float32):
            raise NotImplementedError("Gagorax runs in bfloat16 or float32")
        if self.prefill_portion < 1:
            raise ValueError("prefill_portion must be positive")
        for i, layer in enumerate(self.layers):
            kind, m, mlp = layer["type"], layer["mixer"], layer.get("mlp")
            if kind not in MIXERS:
                raise NotImplementedError("layer %d: unknown mixer %r" % (i, kind))
            missing = [k for k in MIXERS[kind] if k not in m]
            if missing:
                raise ValueError("layer %d: mixer fields missing: %s" % (i, ", ".join(missing)))
            if kind == "attention":
                if m["heads"] % m["kv_heads"]:
                    raise ValueError("layer %d: kv_heads must divide heads" % i)
                if m["rot"]["dims"] % 2 or m["rot"]["dims"] > m["dim"] or m["vdim"] % 2:
                    raise ValueError("layer %d: rotated sizes must be even and fit the head" % i)
            if kind == "lightning" and len(m["decay"]) != m["heads"]:
                raise ValueError("layer %d: one decay per head is required" % i)
            if mlp is not None and mlp["kind"] != "dense":
                raise NotImplementedError("layer %d: unknown feed-forward %r" % (i, mlp["kind"]))

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
