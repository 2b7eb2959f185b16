"""Parts of the Bikelix support that need no device: the oracle's mechanisms against closed forms, windows in the planner, the
configuration."""
import copy

import numpy as np
import pytest

import bikelix_oracle as oracle
from bikelix_cases import CONFIGS, config, latent
from chunk_attn import PrefixTree, cabi
from chunk_attn.models.bikelix import BikelixConfig
from chunk_attn.models.registry import architecture_of


# ---- the oracle ------------------------------------------------------------------------------------------------------

def test_norms():
    x = np.array([[3.0, -4.0]])
    rms = np.sqrt(12.5 + 0.5)  # eps counts inside the root
    assert np.allclose(oracle.plain_norm(x, np.array([2.0, 1.0]), 0.5), [[6 / rms, -4 / rms]])
    assert np.allclose(oracle.centred_norm(x, np.array([1.0, 0.0]), 0.5), oracle.plain_norm(x, np.array([2.0, 1.0]), 0.5))


def test_rotation_pairs_halves_and_is_relative():
    g = np.random.default_rng(0)
    e0 = np.zeros((1, 1, 6))
    e0[0, 0, 1] = 1.0  # pair 1 of 4 rotated elements: elements 1 and 3, frequency base ** (-1/2)
    y = oracle.rotate_halves(e0, [3], 4, 16.0)[0, 0]
    assert np.allclose(y, [0, np.cos(0.75), 0, np.sin(0.75), 0, 0])
    q, k = g.standard_normal((2, 1, 1, 8))
    s = [(oracle.rotate_halves(q, [p + 5], 8, 100.0) * oracle.rotate_halves(k, [p], 8, 100.0)).sum() for p in (0, 3, 50)]
    assert np.allclose(s, s[0])


def test_sink_and_window():
    s = np.array([1.0, 2.0])
    w = oracle.sink_softmax(s, 0.5)
    assert np.allclose(w, np.exp(s) / (np.exp(s).sum() + np.exp(0.5)))
    assert np.allclose(oracle.sink_softmax(s, 800.0), 0)  # finite with a sink far above the scores
    assert list(oracle.window_positions(5, 3)) == [3, 4, 5] and list(oracle.window_positions(1, 3)) == [0, 1]
    assert list(oracle.window_positions(4, 1)) == [4]
    # a window of one token and a negligible sink: the output is the token's own value
    g = np.random.default_rng(1)
    q, k, v = g.standard_normal((3, 4, 2, 5))
    assert np.allclose(oracle.windowed_attention(q, k, v, 0.3, np.full(2, -1e9), 1), v)


def test_clamps_and_soft_cap():
    # the gate is bounded above only, the other half on both sides
    y = oracle.clamped_glu(np.array([9.0, -9.0]), np.array([-7.0, 7.0]), 2.0)
    assert np.allclose(y, [2 / (1 + np.exp(-3.404)) * -1.0, -9 / (1 + np.exp(15.318)) * 3.0])
    assert np.allclose(oracle.softcap(np.array([0.1, 1e6]), 4.0), [4 * np.tanh(0.025), 4.0])


def test_scores_in_the_latent_space_are_the_heads_scores():
    """Folding the key projection into the query and the value projection behind the sum changes nothing."""
    g = np.random.default_rng(2)
    T, H, d, r, dv, R = 6, 3, 4, 2, 5, 7
    c, kr, q = g.standard_normal((T, R)), g.standard_normal((T, r)), g.standard_normal((T, H, d + r))
    U, W, sink = g.standard_normal((H, d, R)), g.standard_normal((H, dv, R)), g.standard_normal(H)
    k = np.concatenate([np.einsum("hdr,tr->thd", U, c), np.broadcast_to(kr[:, None], (T, H, r))], -1)
    want = oracle.windowed_attention(q, k, np.einsum("hdr,tr->thd", W, c), 0.4, sink, 4)
    rows = np.concatenate([c, kr], -1)[:, None].repeat(H, 1)
    ql = np.concatenate([np.einsum("hdr,thd->thr", U, q[..., :d]), q[..., d:]], -1)
    got = np.einsum("hdr,thr->thd", W, oracle.windowed_attention(ql, rows, c[:, None].repeat(H, 1), 0.4, sink, 4))
    assert np.allclose(got, want)


def test_a_reader_uses_the_owners_rows():
    """Changing the owner's key/value projection changes what the reader attends to; the reader's own tensors have none."""
    from chunk_attn.models.bikelix.modeling_bikelix import random_weights
    cfg = config(24, 30, [latent(2, 8, 4, 8, 12, 16, 5), latent(3, 4, 4, 8, 12, 16, 9, kv_from=0)])
    w = {k: v.double().numpy() for k, v in random_weights(BikelixConfig.from_dict(cfg, torch_device="cpu"), 1).items()}
    assert "l1.mix.dkv" not in w and "l1.mix.dkv.norm" not in w
    toks = [1, 5, 7, 9, 2, 4, 8]
    w2 = dict(w, **{"l0.mix.o": w["l0.mix.o"] * 0, "l0.mix.dkv": w["l0.mix.dkv"] * -1.0})
    w3 = dict(w2, **{"l0.mix.dkv": w["l0.mix.dkv"]})
    a, b = oracle.forward(toks, w2, cfg)[1], oracle.forward(toks, w3, cfg)[1]
    assert np.allclose(a[0], b[0]) and not np.allclose(a[1], b[1])


# ---- windows in the planner ---------------------------------------------------------------------------------------------

def tree_of(specs, chunk):
    tree = PrefixTree(chunk_size=chunk, max_chunks=4096)
    rows = []
    for toks in specs:
        rows.insert(tree.add_seq(toks), toks)
    return tree, rows


def paths_of(tree):
    """Per row: [(chunk id, position of its first token, tokens)] from root to leaf."""
    out = []

    def walk(node, at, path):
        path = path + [(node.id, at, node.n_tokens)]
        if not node.children:
            out.append(path)
        for c in node.children:
            walk(c, at + node.n_tokens, path)

    for c in tree.get_trie().children:
        walk(c, 0, [])
    return out


def seen_by_plan(plan, n_rows, chunk, delta):
    """Per row: (chunk id, row in chunk) of every position its items bring, keyed by position."""
    seen = [dict() for _ in range(n_rows)]
    slots = {}
    for it in plan.items():
        n_tiles, first, row_begin, rows, slot_base, flags, last = (int(x) for x in it[:7])
        assert rows >= 1 and first % chunk == 0
        for j in range(n_tiles):
            n = chunk if j < n_tiles - 1 else min(chunk, last + (delta if flags & 1 else 0))
            for r in range(row_begin, row_begin + rows):
                for t in range(n):
                    assert seen[r].setdefault(first + j * chunk + t, (int(it[7 + j]), t)) == (int(it[7 + j]), t)
        for r in range(rows):
            slots.setdefault(row_begin + r, []).append(slot_base + r)
    off, merge = plan.array(cabi.PLAN_MERGE_OFF), plan.array(cabi.PLAN_MERGE_SLOTS)
    for r in range(n_rows):
        assert sorted(merge[off[r]:off[r + 1]].tolist()) == sorted(slots.get(r, []))
    return seen


SHARED = list(range(100, 100 + 40))
SPECS = {
    "alone": [list(range(30))],
    "exact chunks": [list(range(8)), list(range(50, 66))],
    "one prefix": [SHARED + [1000 * s + j for j in range(1 + 9 * s)] for s in range(1, 6)],
    # rows of very different lengths behind the same first chunks, two levels of sharing
    "two levels": [SHARED[:16] + [1] * n for n in (2, 50)] + [SHARED + [2] * n for n in (3, 4, 33)] + [SHARED[:16] + [3, 3, 3, 3] * 4 + [5] * n for n in (1, 20)],
}


@pytest.mark.parametrize("spec", sorted(SPECS))
@pytest.mark.parametrize("window", [1, 3, 4, 5, 16, 17, 37, 1000])
@pytest.mark.parametrize("rows_per_item", [1, 2, 64])
@pytest.mark.parametrize("n_ctas", [1, 8, 296])
def test_windowed_work_lists(spec, window, rows_per_item, n_ctas):
    """Every row's items bring each position of its window exactly from where the tree has it, now and for the tokens that
    follow until the tree changes; chunks before every window are not part of the work."""
    chunk = 4
    tree, rows = tree_of(SPECS[spec], chunk)
    plan = cabi.Plan.windowed(tree.get_chunks(), len(rows), window, chunk_size=chunk, n_ctas=n_ctas, rows_per_item=rows_per_item)
    paths = paths_of(tree)
    assert len(paths) == len(rows)
    room = min(chunk - p[-1][2] for p in paths)
    for delta in range(room + 1):
        seen = seen_by_plan(plan, len(rows), chunk, delta)
        for path, got, toks in zip(paths, seen, rows):
            where = {at + t: (cid, t) for cid, at, n in path for t in range(chunk)}
            last = len(toks) + delta - 1
            for pos in oracle.window_positions(last, window):
                assert got.get(pos) == where[pos], (pos, delta)
            assert all(got[p] == where[p] for p in got)
    # what no row's window (counted from its last stored token) touches is left out
    used = {int(c) for it in plan.items() for c in it[7:7 + int(it[0])]}
    for cid in {c for p in paths for c, _, _ in p}:
        needed = any(c == cid and (at + n > len(t) - window or c == p[-1][0]) for p, t in zip(paths, rows) for c, at, n in p)
        assert (cid in used) == needed


def test_plans_without_a_window_are_unchanged():
    tree, rows = tree_of(SPECS["one prefix"], 4)
    plan = cabi.Plan.windowed(tree.get_chunks(), len(rows), 0, chunk_size=4)
    assert all(int(it[1]) == 0 for it in plan.items())
    with pytest.raises(cabi.CAError):
        cabi.Plan.windowed(tree.get_chunks(), len(rows), -1, chunk_size=4)


# ---- configuration --------------------------------------------------------------------------------------------------

def test_configuration_and_registry():
    assert architecture_of(CONFIGS["odd"]) == "Bikelix"
    for cfg in CONFIGS.values():
        BikelixConfig.from_dict(cfg)
    good = CONFIGS["odd"]

    def broken(change):
        d = copy.deepcopy(good)
        change(d)
        return d

    cases = [(ValueError, lambda d: d["layers"][0]["mixer"].pop("scale")),
             (ValueError, lambda d: d["layers"][0]["mixer"].update(rot_dim=8)),           # not what is rotated
             (ValueError, lambda d: d["layers"][0]["mixer"]["mask"].update(size=0)),
             (ValueError, lambda d: d["layers"][2]["mixer"].update(kv_from=2)),           # itself
             (ValueError, lambda d: d["layers"][3]["mixer"].update(kv_from=2)),           # a reader
             (ValueError, lambda d: d["layers"][3]["mixer"].update(kv_from=0)),           # other sizes
             (ValueError, lambda d: d["layers"][2]["mixer"]["rot"].update(base=3.0)),     # another rotation
             (ValueError, lambda d: d["layers"][0]["mlp"].pop("limit")),
             (ValueError, lambda d: d.update(logit_softcap=0.0)),
             (NotImplementedError, lambda d: d["layers"][0].update(type="other")),
             (NotImplementedError, lambda d: d["layers"][0]["mlp"].update(kind="other"))]
    for error, change in cases:
        with pytest.raises(error):
            BikelixConfig.from_dict(broken(change))
