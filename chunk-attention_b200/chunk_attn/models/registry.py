"""Which classes serve a model folder (config.json + model.safetensors)."""
import json
import os

import torch

from .weights import read_model_weights


def _gagorax(folder, config, dtype, device, engine):
    from .gagorax import GagoraxConfig, GagoraxForCausalLM
    cfg = GagoraxConfig.from_dict(config, torch_dtype=dtype or torch.bfloat16, torch_device=str(device), **engine)
    return GagoraxForCausalLM(cfg, read_model_weights(folder))


def _bikelix(folder, config, dtype, device, engine):
    from .bikelix import BikelixConfig, BikelixForCausalLM
    cfg = BikelixConfig.from_dict(config, torch_dtype=dtype or torch.bfloat16, torch_device=str(device), **engine)
    return BikelixForCausalLM(cfg, read_model_weights(folder))


def _llama(folder, config, dtype, device, engine):
    from .llama_hf import LlamaConfig, LlamaForCausalLM
    dtype = dtype or torch.float16
    cfg = LlamaConfig.from_dict(dict(config, torch_dtype=dtype, torch_device=str(device), **engine))
    model = LlamaForCausalLM(cfg)
    tensors = read_model_weights(folder)
    if "lm_head.weight" not in tensors:  # tied to the embedding
        tensors["lm_head.weight"] = tensors["model.embed_tokens.weight"]
    tensors = {k: v for k, v in tensors.items() if not k.endswith("rotary_emb.inv_freq")}
    model.load_state_dict(tensors)
    return model.to(device=device, dtype=dtype).eval()


MODELS = {"Bikelix": _bikelix, "Gagorax": _gagorax, "LlamaForCausalLM": _llama}


def architecture_of(config):
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    if name not in MODELS:
        raise NotImplementedError("no model of this framework serves architecture %r (known: %s)" % (name, ", ".join(sorted(MODELS))))
    return name


def load_model(folder, dtype=None, device="cuda:0", **engine):
    """The model of a folder, with its weights, on `device`.  engine: fields of the configuration's engine side."""
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    return MODELS[architecture_of(config)](folder, config, dtype, device, engine)
