"""Models from folders: the registry with weights on disk, the trace replay and the command line, for both decoders."""
import io
import json
import struct
import sys

import numpy as np
import pytest
import torch

from chunk_attn import generate, trace
from chunk_attn.models.gagorax import GagoraxConfig
from chunk_attn.models.gagorax.modeling_gagorax import random_weights
from chunk_attn.models.llama_hf import LlamaConfig, LlamaForCausalLM
from chunk_attn.models.registry import load_model
from chunk_attn.models.sequence import Sequence
from gagorax_cases import CONFIGS, TOL, error, reference, tokens_for

pytestmark = pytest.mark.gpu
NAMES = {torch.bfloat16: "BF16", torch.float16: "F16", torch.float32: "F32"}


def write_folder(path, config, tensors):
    (path / "config.json").write_text(json.dumps(config))
    head, at, parts = {}, 0, []
    for name, t in tensors.items():
        t = t.contiguous().cpu()
        raw = t.view(torch.uint8).numpy().tobytes() if t.dim() else t.numpy().tobytes()
        head[name] = {"dtype": NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        at += len(raw)
        parts.append(raw)
    h = json.dumps(head).encode()
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(h)) + h + b"".join(parts))


@pytest.fixture
def gagorax_folder(tmp_path):
    cfg = CONFIGS["odd"]
    w = random_weights(GagoraxConfig.from_dict(cfg), 12)
    (tmp_path / "m").mkdir()
    write_folder(tmp_path / "m", cfg, w)
    return cfg, {k: v.double().numpy() for k, v in w.items()}, tmp_path


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(gagorax_folder, dtype, monkeypatch, capsys):
    cfg, w, path = gagorax_folder
    a, b = tokens_for(cfg, 70, 1), tokens_for(cfg, 40, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[66:67], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[:2], "want": [1]}, {"id": "a", "tokens": a[67:], "want": [0, 2]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b[2:], "want": [37]}], "end": ["b"]},
             {"step": 4, "entries": [{"id": "a", "tokens": b[:5], "want": [4]}], "end": ["a"]}]  # the name is free again
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    out = path / "out"
    out.mkdir()
    assert trace.main(["--model", str(path / "m"), "--dtype", dtype, "--out", str(out), "--max-tokens", "200"]) == 0
    assert [l for l in capsys.readouterr().out.splitlines() if l.startswith("done")] == ["done %d" % i for i in range(5)]
    assert sorted(p.name for p in out.iterdir()) == ["0.f32", "2.f32", "3.f32", "4.f32"]
    ra, rb = reference(cfg, w, a), reference(cfg, w, b)
    want = {0: ra[[0, 65]], 2: np.stack([rb[1], ra[67], ra[69]]), 3: rb[[39]], 4: rb[[4]]}
    for step, ref in want.items():
        got = np.fromfile(out / ("%d.f32" % step), "<f4").reshape(ref.shape)
        assert error(got, ref) < TOL[getattr(torch, dtype)], step


def test_generation_command(gagorax_folder, monkeypatch, capsys):
    cfg, w, path = gagorax_folder
    prompts = [tokens_for(cfg, n, n) for n in (3, 70)]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(" ".join(map(str, p)) for p in prompts) + "\n"))
    assert generate.main(["--model", str(path / "m"), "--dtype", "float32", "--max-new-tokens", "6"]) == 0
    lines = [[int(t) for t in l.split()] for l in capsys.readouterr().out.splitlines()]
    assert [len(l) for l in lines] == [9, 76]
    for p, toks in zip(prompts, lines):
        assert toks[:len(p)] == p
        ref = reference(cfg, w, toks)
        for t in range(len(p) - 1, len(toks) - 1):
            assert ref[t, toks[t + 1]] >= ref[t].max() - 1e-3


def test_llama_from_a_folder(tmp_path):
    fields = {"vocab_size": 64, "hidden_size": 128, "intermediate_size": 96, "num_hidden_layers": 2, "num_attention_heads": 2,
              "max_position_embeddings": 128}
    direct = LlamaForCausalLM(LlamaConfig(torch_device="cuda:0", chunk_attn_kvcache_gb=0.1, **fields), seed=3).to("cuda:0", torch.float16)
    write_folder(tmp_path, dict(fields, architectures=["LlamaForCausalLM"]), direct.state_dict())
    model = load_model(str(tmp_path), chunk_attn_kvcache_gb=0.1)
    toks = [5, 9, 33, 2]
    assert torch.equal(model.logits([Sequence(toks)], None, True), direct.logits([Sequence(toks)], None, True))


def test_unknown_tokens_are_refused(gagorax_folder):
    cfg, w, path = gagorax_folder
    model = load_model(str(path / "m"))
    caches = model.create_kv_caches(max_tokens=64)
    with pytest.raises(RuntimeError, match="vocabulary"):
        model.step([None], [[cfg["vocab"]]], caches)
