"""Weights on disk: a reader of safetensors files (an 8-byte little-endian length, that many bytes of JSON, the raw
tensors).  Tensors are views of the memory-mapped file until they are moved to a device."""
import json
import mmap
import os
import struct

import torch

DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
          "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_safetensors(path):
    """{name: CPU tensor} of one file."""
    with open(path, "rb") as f:
        buf = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    n = struct.unpack("<Q", buf[:8])[0]
    if 8 + n > len(buf):
        raise ValueError("%s: truncated header" % path)
    header = json.loads(buf[8:8 + n])
    out = {}
    for name, spec in header.items():
        if name == "__metadata__":
            continue
        lo, hi = spec["data_offsets"]
        dtype = DTYPES[spec["dtype"]]
        count = 1
        for s in spec["shape"]:
            count *= s
        if hi - lo != count * dtype.itemsize or 8 + n + hi > len(buf):
            raise ValueError("%s: tensor %s does not fit its place in the file" % (path, name))
        if count == 0:
            out[name] = torch.empty(spec["shape"], dtype=dtype)
            continue
        out[name] = torch.frombuffer(buf, dtype=dtype, count=count, offset=8 + n + lo).reshape(spec["shape"])
    return out


def read_model_weights(folder):
    """All tensors of a model folder: model.safetensors, or the shards model.safetensors.index.json names."""
    index = os.path.join(folder, "model.safetensors.index.json")
    if os.path.exists(index):
        with open(index) as f:
            shards = sorted(set(json.load(f)["weight_map"].values()))
    else:
        shards = ["model.safetensors"]
    out = {}
    for s in shards:
        out.update(read_safetensors(os.path.join(folder, s)))
    return out
