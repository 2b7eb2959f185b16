"""The Bikelix decoder on the GPU against its plain oracle: whole prompts, portions, decoding, mixed batches, reuse of
chunks, keys on the edges of windows, model folders, and greedy generation through the host."""
import io
import json
import random
import sys

import numpy as np
import pytest
import torch

import bikelix_oracle as oracle
import chunk_attn.models.bikelix.modeling_bikelix as modeling
from bikelix_cases import CONFIGS, TOL, Driver, config, error, latent, make, random_weights, reference, tokens_for
from chunk_attn import generate, trace
from chunk_attn.models.bikelix import BikelixConfig
from chunk_attn.models.model_host import ModelHost
from chunk_attn.models.sequence import Sequence
from test_gpu_gagorax import cuts
from test_gpu_model_folders import write_folder

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture
def paths(monkeypatch):
    """Counts which of its two forms attention has taken: [in the latent space, expanded]."""
    count = [0, 0]
    chosen = modeling.LatentAttentionMixer.expands

    def counted(self, *a):
        r = chosen(self, *a)
        count[r] += 1
        return r

    monkeypatch.setattr(modeling.LatentAttentionMixer, "expands", counted)
    return count


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(name, dtype, paths):
    cfg = CONFIGS[name]
    model, w = make(cfg, dtype, seed=1)
    d = Driver(model)
    for i, n in enumerate((1, 2, 63, 64, 65, 128, 200)):
        toks = tokens_for(cfg, n, i)
        d.step([("r%d" % i, toks)])
        d.end("r%d" % i)
        assert error(d.logits("r%d" % i), reference(cfg, w, toks)) < TOL[dtype], n
    assert d.clean()
    assert (paths[1] > 0) == (dtype == torch.bfloat16 and name != "odd")  # its head sizes are no whole granules


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_stream_after_every_layer(name, dtype):
    cfg = CONFIGS[name]
    model, w = make(cfg, dtype, seed=11)
    toks = tokens_for(cfg, 90, 3)
    got = []
    model.step([None], [toks], model.create_kv_caches(max_tokens=256), tap=lambda i, x: got.append(x.cpu().numpy().copy()))
    want = oracle.forward(toks, w, cfg)[1]
    assert len(got) == len(cfg["layers"])
    for i, (g, x) in enumerate(zip(got, want)):
        assert np.abs(g - x).max() < (2e-5 if dtype == torch.float32 else 0.15), i


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_token_by_token_and_portions(name, dtype):
    """The same tokens whole, one by one, and in portions down to two tokens, cut anywhere."""
    cfg = CONFIGS[name]
    model, w = make(cfg, dtype, seed=2)
    toks = tokens_for(cfg, 250, 7)
    want = reference(cfg, w, toks)
    for sizes in ([1], [2], [3, 2, 61, 1, 2, 64], [64], [130, 1, 1, 2, 37]):
        d = Driver(model)
        at = 0
        for n in cuts(len(toks), sizes):
            d.step([("a", toks[at:at + n])])
            at += n
        assert error(d.logits("a"), want) < TOL[dtype], sizes
        assert d.clean()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "wide", "large"])
def test_batches_of_unequal_requests(name, dtype):
    """Requests that start, continue and decode in the same steps get what each gets alone; chunks that finished
    requests leave are used again, and a request that shares a long prefix reads another's chunks."""
    cfg = CONFIGS[name]
    model, w = make(cfg, dtype, seed=3)
    rnd = random.Random(5)
    shared = tokens_for(cfg, 130, 50)
    todo = {"s%d" % i: shared + tokens_for(cfg, 5 + 30 * i, 60 + i) for i in range(3)}
    todo.update({"u%d" % i: tokens_for(cfg, n, 70 + i) for i, n in enumerate((1, 7, 64, 190, 3, 90, 128, 66))})
    names = list(todo)
    rnd.shuffle(names)
    d = Driver(model, max_tokens=1200)
    at, live = {n: 0 for n in names}, []
    while names or live:
        while names and len(live) < 4:
            live.append(names.pop())
        # some requests rest in a step; a step in which all live ones bring one token is a decode step
        one = rnd.random() < 0.4
        picked = live if one and all(at[n] for n in live) else [n for n in live if rnd.random() < 0.8] or live[:1]
        entries = []
        for n in picked:
            k = 1 if one or rnd.random() < 0.3 else rnd.choice([2, 3, 17, 64, 100])
            entries.append((n, todo[n][at[n]:at[n] + k]))
        if entries and all(at[n] for n, _ in entries):  # decode steps come in row order
            entries.sort(key=lambda e: d.order.index(e[0]))
        d.step(entries)
        for n, t in entries:
            at[n] += len(t)
            if at[n] == len(todo[n]):
                d.end(n)
                live.remove(n)
    for n, toks in todo.items():
        assert error(d.logits(n), reference(cfg, w, toks)) < TOL[dtype], n
    assert d.clean() and not d.order


@pytest.mark.parametrize("dtype", DTYPES)
def test_decoding_batch_over_a_shared_prefix(dtype):
    """Many rows decode together over a prefix they share, beyond the end of windows and chunks; the owner's and the readers'
    work lists are made once for all layers of a kind."""
    cfg = CONFIGS["wide"]
    model, w = make(cfg, dtype, seed=4)
    d = Driver(model, max_tokens=8192)
    shared = tokens_for(cfg, 192, 1)
    toks = {"r%d" % i: shared + tokens_for(cfg, 3 + (7 * i) % 70, 10 + i) for i in range(9)}
    extra = {n: tokens_for(cfg, 70, 100 + i) for i, n in enumerate(toks)}
    for n, t in toks.items():
        d.step([(n, t)])
    for k in range(70):
        d.step([(n, [extra[n][k]]) for n in d.order])
    if dtype == torch.bfloat16:
        stats = d.caches[0].plan_stats()
        assert stats["n_runs"] >= 1 and stats["n_shared_chunks"] >= 1
    for n in toks:
        assert error(d.logits(n), reference(cfg, w, toks[n] + extra[n])) < TOL[dtype], n
    assert d.clean()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    cfg = config(64, 50, [latent(4, 16, 16, 16, 24, 48, 100, ff=64), latent(3, 24, 16, 8, 24, 48, 300, kv_from=0)])
    model, w = make(cfg, dtype, seed=5)
    toks = tokens_for(cfg, 700, 3)
    d = Driver(model)
    d.step([("a", toks[:5])])
    for t in toks[5:]:
        d.step([("a", [t])])
    assert error(d.logits("a"), reference(cfg, w, toks)) < TOL[dtype]


def sharp_weights(cfg, w, layer, owner):
    """Makes token 1's key stand out for token 0's query in `layer`, whose rows layer `owner` stores: both tokens' streams are
    one large element each, which the latents keep, and the heads' first unrotated element carries it into the score."""
    w = {k: v.clone() for k, v in w.items()}
    m = cfg["layers"][layer]["mixer"]
    p, o = "l%d.mix." % layer, "l%d.mix." % owner
    for tok in (0, 1):
        w["embed"][tok].zero_()
        w["embed"][tok, tok] = 8.0
    for name, key in ((p + "dq", 0), (o + "dkv", 1)):
        w[name][:, 0] = 0.0
        w[name][:, 1] = 0.0
        w[name][0] = 0.0
        w[name][0, key] = 4.0
    R, q_rank = m["kv_rank"], m["q_rank"]
    w[o + "dkv"][1:R + m["rot_dim"], 1] = 0.0  # token 1: the latent is its first element alone, the rotated part is zero
    w[o + "dkv.norm"].fill_(1.0)
    w[p + "dq.norm"].fill_(1.0)
    uq, uk = w[p + "uq"].view(m["heads"], m["dim"] + m["rot_dim"], q_rank), w[p + "uk"].view(m["heads"], m["dim"], R)
    uq[:, :, 0] = 0.0
    uk[:, :, 0] = 0.0
    uq[:, 0, 0] = 4.0
    uk[:, 0, 0] = 4.0
    # score = 4 sqrt(q_rank) * 4 sqrt(R) * scale
    w[p + "sink"].zero_()
    w[p + "sink"][0] = 10.0
    return w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("reader", [False, True])
@pytest.mark.parametrize("window", [41, 64, 150])
def test_keys_on_the_edge_of_a_window(dtype, reader, window):
    """One key that dwarfs all others, just inside the window (it decides the logits) and just outside (it must not be seen): in
    a prompt, in a portion of two tokens, and decoded; in a layer with rows of its own and in one that reads another's."""
    m = dict(heads=4, dim=16, rot=16, vdim=24, q_rank=24, kv_rank=40, window=window, scale=0.06)
    layers = [latent(4, 16, 16, 24, 24, 40, 30), latent(kv_from=0, **m)] if reader else [latent(**m)]
    cfg = config(80, 40, layers, alpha=0.5)
    base = random_weights(BikelixConfig.from_dict(cfg), 6)
    if reader:  # nothing but the embedding reaches the second layer
        base["l0.mix.o"].zero_()
    model, w = make(cfg, dtype, weights=sharp_weights(cfg, base, len(layers) - 1, 0))
    for inside in (True, False):
        distance = window - 1 if inside else window
        n = distance + 4
        toks = [t % 38 + 2 for t in tokens_for(cfg, n, distance)]
        toks[n - 1 - distance], toks[n - 1] = 1, 0
        want = reference(cfg, w, toks)
        other = list(toks)
        other[n - 1 - distance] = 5
        assert (error(reference(cfg, w, other)[-1:], want[-1:]) > 0.3) == inside  # the key matters exactly when it is seen
        d = Driver(model)
        d.step([("whole", toks)])
        d.end("whole")
        d.step([("dec", toks[:-1])])
        d.step([("dec", toks[-1:])])
        d.end("dec")
        d.step([("two", toks[:-2])])
        d.step([("two", toks[-2:])])
        for name in ("whole", "dec", "two"):
            assert error(d.logits(name)[-1:], want[-1:]) < TOL[dtype], (name, inside)


@pytest.mark.parametrize("dtype", DTYPES)
def test_generation_through_the_host(dtype):
    """Greedy generation with arrivals, more requests than rows and prompts run in portions: every token chosen is the
    oracle's best one, up to rounding."""
    cfg = CONFIGS["odd" if dtype == torch.float32 else "wide"]
    model, w = make(cfg, dtype, seed=8, prefill_portion=50, kvcache_gb=0.25, state_slots=2)
    shared = tokens_for(cfg, 70, 20)
    prompts = [shared + tokens_for(cfg, n, 30 + n) for n in (3, 40)] + [tokens_for(cfg, n, 40 + n) for n in (1, 64, 120, 17)]
    lens = [20, 5, 12, 1, 30, 9]
    host = ModelHost(model, model.create_kv_caches(), max_batch_size=3)
    host.cycle_time = 0.05
    with host:
        pending = [host.predict_async(p, n) for p, n in zip(prompts, lens)]
        results = [s.get_result(timeout=120) for s in pending]
    assert host.peak_batch_size <= 3
    slack = 4 * TOL[dtype]
    for p, n, toks in zip(prompts, lens, results):
        assert toks[:len(p)] == p and len(toks) == len(p) + n
        ref = reference(cfg, w, toks)
        for t in range(len(p) - 1, len(toks) - 1):
            assert ref[t, toks[t + 1]] >= ref[t].max() - slack * ref.std(), t
    assert len(host.kv_caches[-1]) == 0 and all(len(c.get_trie().children) == 0 for c in host.kv_caches[:-1])


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_of_any_budget_give_the_same_prompt(dtype):
    cfg = CONFIGS["large"]
    prompts = [tokens_for(cfg, n, n) for n in (5, 100, 1, 270)]
    outs = []
    for budget in (2, 37, 8192):
        model, w = make(cfg, dtype, seed=9, prefill_portion=budget, kvcache_gb=0.25)
        seqs = [Sequence(p) for p in prompts]
        outs.append(model.logits(seqs, model.create_kv_caches(), prefill=True).cpu().numpy())
        assert [s.index is not None for s in seqs] == [True] * 4
    want = np.stack([reference(cfg, w, p)[-1] for p in prompts])
    for o in outs:
        assert error(o, want) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_caches_of_any_chunk_size(dtype):
    """Chunks the tensor-core kernels do not take: every step runs as portions of the any-geometry kernel."""
    cfg = CONFIGS["odd"]
    model, w = make(cfg, dtype, seed=13, chunk_size=8)
    toks = tokens_for(cfg, 60, 2)
    d = Driver(model)
    d.step([("a", toks[:41])])
    for t in toks[41:]:
        d.step([("a", [t])])
    assert error(d.logits("a"), reference(cfg, w, toks)) < TOL[dtype]


def test_a_refused_step_changes_nothing():
    cfg = CONFIGS["wide"]
    model, w = make(cfg, torch.bfloat16, seed=10)
    small = Driver(model, max_tokens=64)
    with pytest.raises(RuntimeError, match="capacity"):
        small.step([("big", tokens_for(cfg, 600000, 1))])
    toks = [1, 2, 3]
    small.step([("ok", toks)])
    assert error(small.logits("ok"), reference(cfg, w, toks)) < TOL[torch.bfloat16]
    with pytest.raises(RuntimeError, match="vocabulary"):
        model.step([None], [[cfg["vocab"]]], model.create_kv_caches(max_tokens=64))


# ---- from folders ------------------------------------------------------------------------------------------------------

@pytest.fixture
def folder(tmp_path):
    cfg = CONFIGS["odd"]
    w = random_weights(BikelixConfig.from_dict(cfg), 12)
    (tmp_path / "m").mkdir()
    write_folder(tmp_path / "m", cfg, w)
    return cfg, {k: v.double().numpy() for k, v in w.items()}, tmp_path


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(folder, dtype, monkeypatch, capsys):
    cfg, w, path = folder
    a, b = tokens_for(cfg, 70, 1), tokens_for(cfg, 40, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[66:67], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[:2], "want": [1]}, {"id": "a", "tokens": a[67:], "want": [0, 2]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b[2:], "want": [37]}], "end": ["b"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    out = path / "out"
    out.mkdir()
    assert trace.main(["--model", str(path / "m"), "--dtype", dtype, "--out", str(out), "--max-tokens", "200"]) == 0
    assert [l for l in capsys.readouterr().out.splitlines() if l.startswith("done")] == ["done %d" % i for i in range(4)]
    ra, rb = reference(cfg, w, a), reference(cfg, w, b)
    for step, ref in {0: ra[[0, 65]], 2: np.stack([rb[1], ra[67], ra[69]]), 3: rb[[39]]}.items():
        got = np.fromfile(out / ("%d.f32" % step), "<f4").reshape(ref.shape)
        assert error(got, ref) < TOL[getattr(torch, dtype)], step


def test_generation_command(folder, monkeypatch, capsys):
    cfg, w, path = folder
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
