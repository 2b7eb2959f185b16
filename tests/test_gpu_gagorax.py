"""The Gagorax decoder on the GPU against its plain oracle: whole prompts, portions, decoding, mixed batches, reuse of
chunks and slots, and greedy generation through the host."""
import random

import numpy as np
import pytest
import torch

from chunk_attn.models.model_host import ModelHost
from chunk_attn.models.sequence import Sequence
from gagorax_cases import CONFIGS, TOL, Driver, attention, config, error, lightning, make, mamba, reference, tokens_for

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def cuts(total, sizes):
    out, k = [], 0
    while total:
        n = min(total, sizes[k % len(sizes)])
        out.append(n)
        total -= n
        k += 1
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(name, dtype):
    cfg = CONFIGS[name]
    model, w = make(cfg, dtype, seed=1)
    d = Driver(model)
    for i, n in enumerate((1, 2, 63, 64, 65, 128, 200)):
        toks = tokens_for(cfg, n, i)
        d.step([("r%d" % i, toks)])
        d.end("r%d" % i)
        assert error(d.logits("r%d" % i), reference(cfg, w, toks)) < TOL[dtype], n
    assert d.clean()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_token_by_token_and_portions(name, dtype):
    """The same tokens whole, one by one, and in portions down to two tokens, cut anywhere."""
    cfg = CONFIGS[name]
    model, w = make(cfg, dtype, seed=2)
    toks = tokens_for(cfg, 150, 7)
    want = reference(cfg, w, toks)
    for sizes in ([1], [2], [3, 2, 61, 1, 2, 64], [64], [100, 1, 1, 2]):
        d = Driver(model)
        at = 0
        for n in cuts(len(toks), sizes):
            d.step([("a", toks[at:at + n])])
            at += n
        assert error(d.logits("a"), want) < TOL[dtype], sizes
        assert d.clean()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "grouped", "recurrent"])
def test_batches_of_unequal_requests(name, dtype):
    """Requests that start, continue and decode in the same steps get what each gets alone; chunks and slots that
    finished requests leave are used again, and a request that shares a long prefix reads another's chunks."""
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
    """Many rows decode together over a prefix they share: the decode kernels walk it once for all of them."""
    cfg = CONFIGS["grouped"]
    model, w = make(cfg, dtype, seed=4)
    d = Driver(model, max_tokens=8192)
    shared = tokens_for(cfg, 192, 1)
    toks = {"r%d" % i: shared + tokens_for(cfg, 3 + (7 * i) % 70, 10 + i) for i in range(9)}
    extra = {n: tokens_for(cfg, 70, 100 + i) for i, n in enumerate(toks)}
    for n, t in toks.items():
        d.step([(n, t)])
    for k in range(70):
        d.step([(n, [extra[n][k]]) for n in d.order])
    stats = d.caches[0].plan_stats()
    assert stats["n_chunks"] > 0
    for n in toks:
        assert error(d.logits(n), reference(cfg, w, toks[n] + extra[n])) < TOL[dtype], n
    assert d.clean()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    cfg = config(64, 50, [attention(4, 2, 32, 16, 16, ff=64), mamba(64, 16, 4, 4), lightning(32, 16, [0.999, 0.9])])
    model, w = make(cfg, dtype, seed=5)
    toks = tokens_for(cfg, 700, 3)
    d = Driver(model)
    d.step([("a", toks[:5])])
    for t in toks[5:]:
        d.step([("a", [t])])
    assert error(d.logits("a"), reference(cfg, w, toks)) < TOL[dtype]


def sharp_weights(cfg, w, layer):
    """Makes one key of `layer` stand out for one query: token 1's key direction equals token 0's query direction."""
    w = {k: v.clone() for k, v in w.items()}
    p = "l%d." % layer
    m = cfg["layers"][layer]["mixer"]
    W = cfg["width"]
    w["embed"][0].zero_()
    w["embed"][1].zero_()
    w["embed"][0, 0] = 8.0
    w["embed"][1, 1] = 8.0
    w[p + "shift"].zero_()
    for name, col in (("q", 0), ("k", 1)):
        a = w[p + "mix." + name].view(-1, m["dim"], W)
        a[:, :, col] = 0.0
        a[:, m["dim"] - 1, col] = 4.0  # a dimension that is not rotated: the score does not depend on the distance
        other = [0, 1][1 - col]
        a[:, m["dim"] - 1, other] = 0.0
        w[p + "mix." + name + ".norm"].fill_(1.0)
    return w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("distance", [1, 2, 63, 64, 65, 127, 128, 300])
def test_one_far_key_among_many(dtype, distance):
    """A query whose score with ONE key, `distance` tokens back, dwarfs all others: at chunk borders and far away, in a
    prompt and decoded.  Losing or misplacing that key changes the logits."""
    cfg = config(80, 40, [attention(4, 2, 24, 16, 16, scale=1.0), mamba(64, 4, 4, 2)])
    from chunk_attn.models.gagorax import GagoraxConfig
    from chunk_attn.models.gagorax.modeling_gagorax import random_weights
    base = random_weights(GagoraxConfig.from_dict(cfg), 6)
    model, w = make(cfg, dtype, weights=sharp_weights(cfg, base, 0))
    n = distance + 4
    toks = [t % 38 + 2 for t in tokens_for(cfg, n, distance)]
    toks[n - 1 - distance] = 1
    toks[n - 1] = 0
    want = reference(cfg, w, toks)
    other = list(toks)
    other[n - 1 - distance] = 5
    assert error(reference(cfg, w, other)[-1:], want[-1:]) > 0.3  # the key matters
    d = Driver(model)
    d.step([("whole", toks)])
    d.end("whole")
    d.step([("dec", toks[:-1])])
    d.step([("dec", toks[-1:])])
    d.end("dec")
    d.step([("two", toks[:-2])])
    d.step([("two", toks[-2:])])
    for name in ("whole", "dec", "two"):
        assert error(d.logits(name)[-1:], want[-1:]) < TOL[dtype], name


@pytest.mark.parametrize("dtype", DTYPES)
def test_generation_through_the_host(dtype):
    """Greedy generation with arrivals, more requests than rows and prompts run in portions: every token chosen is the
    oracle's best one, up to rounding."""
    cfg = CONFIGS["odd"]
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


def test_portions_of_any_budget_give_the_same_prompt():
    cfg = CONFIGS["grouped"]
    prompts = [tokens_for(cfg, n, n) for n in (5, 100, 1, 70)]
    outs = []
    for budget in (2, 37, 8192):
        model, w = make(cfg, torch.float32, seed=9, prefill_portion=budget, kvcache_gb=0.25)
        seqs = [Sequence(p) for p in prompts]
        outs.append(model.logits(seqs, model.create_kv_caches(), prefill=True).cpu().numpy())
        assert [s.index is not None for s in seqs] == [True] * 4
    want = np.stack([reference(cfg, w, p)[-1] for p in prompts])
    for o in outs:
        assert error(o, want) < TOL[torch.float32]


def test_slots_grow_and_a_failed_step_reports():
    cfg = CONFIGS["recurrent"]
    model, w = make(cfg, torch.float32, seed=10, state_slots=1)
    d = Driver(model)
    toks = [tokens_for(cfg, 9, i) for i in range(5)]
    for i, t in enumerate(toks):
        d.step([(i, t[:4])])
    d.step([(i, t[4:]) for i, t in enumerate(toks)])
    for i, t in enumerate(toks):
        assert error(d.logits(i), reference(cfg, w, t)) < TOL[torch.float32]
    model, _ = make(CONFIGS["grouped"], torch.bfloat16, seed=10)
    small = Driver(model, max_tokens=64)
    with pytest.raises(RuntimeError, match="capacity"):
        small.step([("big", tokens_for(CONFIGS["grouped"], 600000, 1))])
    small.step([("ok", [1, 2, 3])])  # a refused step changed nothing


def test_the_decoder_refuses_what_it_cannot_serve():
    from chunk_attn.models.gagorax import GagoraxConfig
    bad = config(64, 50, [attention(4, 3, 32, 16, 16)])
    with pytest.raises(ValueError):
        GagoraxConfig.from_dict(bad)
    with pytest.raises(NotImplementedError):
        GagoraxConfig.from_dict(config(64, 50, [dict(mamba(8, 2, 2, 2), type="other")]))
    with pytest.raises(NotImplementedError):
        GagoraxConfig.from_dict(config(64, 50, [mamba(8, 2, 2, 2)]), torch_dtype=torch.float16)
