"""Parts of the Gagorax support that need no device: the oracle against step-by-step definitions, portions in the prefix
tree, the recurrent-state rows, weights on disk, the registry."""
import json
import struct

import numpy as np
import pytest
import torch

import gagorax_oracle as oracle
from chunk_attn import PrefixTree, SpanBatch
from chunk_attn.models.recurrent_state import RecurrentState
from chunk_attn.models.registry import architecture_of
from chunk_attn.models.weights import read_model_weights, read_safetensors


def test_oracle_states_carry_over():
    """The recurrences run in two parts from the first part's end state give the whole's outputs."""
    g = np.random.default_rng(0)
    x, dt = g.standard_normal((20, 6)), np.abs(g.standard_normal((20, 6)))
    A, B, C, D = -np.abs(g.standard_normal((6, 3))), g.standard_normal((20, 3)), g.standard_normal((20, 3)), g.standard_normal(6)
    y, S = oracle.selective_scan(x, dt, A, B, C, D)
    y1, S1 = oracle.selective_scan(x[:7], dt[:7], A, B[:7], C[:7], D)
    y2, S2 = oracle.selective_scan(x[7:], dt[7:], A, B[7:], C[7:], D, S1)
    assert np.allclose(np.concatenate([y1, y2]), y) and np.allclose(S, S2)
    q, k, v = g.standard_normal((3, 15, 2, 4))
    o, S = oracle.decayed_linear_attention(q, k, v, [0.5, 0.9])
    for i in range(15):  # the closed form
        w = np.array([0.5, 0.9])[None] ** np.arange(i, -1, -1)[:, None]
        want = np.einsum("hd,jhd,jh,jhe->he", q[i], k[:i + 1], w, v[:i + 1])
        assert np.allclose(o[i], want)


def test_oracle_rotation_is_relative():
    """Scores of rotated q and k depend on the distance only, and turning values forth and back by the same position is the
    identity."""
    g = np.random.default_rng(1)
    q, k = g.standard_normal((2, 1, 1, 8))
    s = [(oracle.rotary(q, [p + 5], 6, 100.0) * oracle.rotary(k, [p], 6, 100.0)).sum() for p in (0, 3, 50)]
    assert np.allclose(s, s[0])
    assert np.allclose(oracle.rotary(oracle.rotary(q, [9], 8, 100.0), [-9], 8, 100.0), q)
    # pair 0 turns by the position itself
    assert np.allclose(oracle.rotary(np.array([[[1.0, 0.0, 0.0, 0.0]]]), [2], 4, 7.0)[0, 0, :2], [np.cos(2), np.sin(2)])


def test_oracle_sink():
    q, k, v = np.ones((1, 1, 2)), np.ones((1, 1, 2)), np.full((1, 1, 3), 5.0)
    assert np.allclose(oracle.sink_attention(q, k, v, 0.5), 5 * np.e / (1 + np.e))


def path_tokens(tree, row):
    """Tokens along the path to row `row`'s tail, found from the root."""
    rows = []

    def walk(node, prefix):
        here = prefix + list(node.tokens)
        if not node.children:
            rows.append(here)
        for c in node.children:
            walk(c, here)

    for c in tree.get_trie().children:
        walk(c, [])
    return rows[row]


@pytest.mark.parametrize("sizes", [[1] * 23, [2, 3, 4, 5, 9], [4, 4, 4, 11], [8, 8, 7], [23]])
def test_portions_in_the_prefix_tree(sizes):
    tree = PrefixTree(chunk_size=4, max_chunks=64)
    toks = list(range(100, 100 + sum(sizes)))
    at, place = 0, {}
    for n in sizes:
        part = toks[at:at + n]
        if at == 0:
            row, created = tree.add_seq_detailed(part)
            assert row == 0
            for cid, start, cnt in created:
                for j in range(cnt):
                    place[start + j] = (cid, j)
        else:
            for i, s in enumerate(tree.extend_seq(0, part)):
                place[at + i] = s
        at += n
        assert path_tokens(tree, 0) == toks[:at]
        assert tree.tails[0].n_tokens < 4  # the tail always has room
    assert len(set(place.values())) == len(toks)  # every token has a row of its own
    assert all(place[t][1] == t % 4 for t in place)
    # a later prompt shares the full chunks the portions made
    row, created = tree.add_seq_detailed(toks[:16] + [1, 2])
    assert created[0][1] == 16
    tree.clear()
    assert tree.chunks_in_use() == 0


def test_portions_respect_the_capacity():
    tree = PrefixTree(chunk_size=4, max_chunks=3)
    tree.add_seq([1, 2])
    with pytest.raises(RuntimeError, match="capacity"):
        tree.extend_seq(0, list(range(10)))  # would leave a full last chunk: needs a fourth
    assert path_tokens(tree, 0) == [1, 2] and tree.chunks_in_use() == 1
    tree.extend_seq(0, list(range(9)))
    assert tree.chunks_in_use() == 3
    with pytest.raises(RuntimeError):
        tree.extend_seq(1, [1])


def test_recurrent_state_rows():
    s = RecurrentState("cpu", slots=2)
    s.register("a", (3,))
    assert s.insert(0) == 0 and s.insert(0) == 1 and s.rows == [1, 0]
    s["a"][1] = 5.0
    s.length[1] = 9
    assert s.insert(2) == 2 and s.capacity == 4 and s["a"].shape == (4, 3) and float(s["a"][1, 0]) == 5.0
    s.remove_seq(0)
    assert s.rows == [0, 2] and s.free == [1, 3] and len(s) == 2
    s["a"][2] = 7.0
    s.length[2] = 4
    s.duplicate(1, 1)  # the lowest free slot, right after its source
    assert s.rows == [0, 2, 1] and s.length[1] == 4 and float(s["a"][1, 2]) == 7.0
    with pytest.raises(IndexError):
        s.insert(7)
    s.clear()
    assert s.free == [0, 1, 2, 3] and not s.length


def test_span_batch_tables():
    sp = SpanBatch([[7, 8, 9], [5], [1, 2]], [4, 0, 10], [3, 0, 1], torch.device("cpu"), work_len=2)
    assert (sp.n_entries, sp.n_tokens, sp.single) == (3, 6, False)
    assert sp.tokens.tolist() == [7, 8, 9, 5, 1, 2] and sp.positions.tolist() == [4, 5, 6, 0, 10, 11]
    assert sp.entry_of.tolist() == [0, 0, 0, 1, 2, 2] and sp.last.tolist() == [2, 3, 5]
    for bad in (([[1], [2]], [0, 0], [1, 1]), ([[]], [0], [0]), ([[1]], [-1], [0]), ([], [], [])):
        with pytest.raises(RuntimeError):
            SpanBatch(*bad, torch.device("cpu"))


def write_safetensors(path, tensors):
    head, data = {"__metadata__": {"format": "pt"}}, b""
    for name, (dtype, shape, raw) in tensors.items():
        head[name] = {"dtype": dtype, "shape": shape, "data_offsets": [len(data), len(data) + len(raw)]}
        data += raw
    h = json.dumps(head).encode()
    path.write_bytes(struct.pack("<Q", len(h)) + h + data)


def test_weights_on_disk(tmp_path):
    a = torch.arange(6).to(torch.bfloat16).reshape(2, 3)
    write_safetensors(tmp_path / "model.safetensors",
                      {"a": ("BF16", [2, 3], a.view(torch.int16).numpy().tobytes()), "i": ("I32", [2], np.array([4, -1], np.int32).tobytes()),
                       "e": ("F32", [0, 4], b"")})
    t = read_model_weights(str(tmp_path))
    assert torch.equal(t["a"], a) and t["i"].tolist() == [4, -1] and t["e"].shape == (0, 4)
    write_safetensors(tmp_path / "bad.safetensors", {"a": ("F32", [3], b"\0" * 8)})
    with pytest.raises(ValueError):
        read_safetensors(str(tmp_path / "bad.safetensors"))


def test_registry_names():
    assert architecture_of({"architecture": "Gagorax"}) == "Gagorax"
    assert architecture_of({"architectures": ["LlamaForCausalLM"]}) == "LlamaForCausalLM"
    with pytest.raises(NotImplementedError):
        architecture_of({"architecture": "Unknown"})
