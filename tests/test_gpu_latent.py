"""Latent caches and the block kernels beside them, one mechanism at a time, against the plain oracle.  Queries are aimed: each
one's best key dwarfs the others and lies at a chosen distance, so that a window that is one token off, a page read from the
wrong place or a sink left out shows."""
import numpy as np
import pytest
import torch

import bikelix_oracle as oracle
import chunk_attn
from chunk_attn import SpanBatch, ops

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")
DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 2e-5, torch.bfloat16: 1.2e-2}


def rnd(seed, *shape, scale=1.0):
    return torch.from_numpy(np.random.default_rng(seed).standard_normal(shape).astype(np.float32) * scale)


def f64(t):
    return t.detach().double().cpu().numpy()


def close(got, want, dtype, what=""):
    err = np.abs(f64(got) - want).max() / max(1.0, np.abs(want).max())
    assert err <= TOL[dtype], "%s: %g" % (what, err)


# ---- block kernels -----------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W", [(1, 64), (5, 97), (3, 1000), (2, 4096), (700, 72), (1, 9001)])
def test_scaled_norm(dtype, T, W):
    x, r, w, b = rnd(1, T, W).to(DEV), rnd(2, T, W, scale=3.0).to(DEV, dtype), (rnd(3, W) * 0.2).to(DEV), rnd(4, W).to(DEV)
    for bias in (None, b):
        y = x.clone()
        plain = ops.scaled_norm(y, r, 1.7, w + 1.0, 0.3, bias=bias)  # a large eps shows where it is added
        want = oracle.centred_norm(1.7 * f64(x) + f64(r) + (f64(b) if bias is not None else 0.0), f64(w), 0.3)
        close(y, want, torch.float32, "stream")
        close(plain, want, dtype, "rounded")
        assert plain.dtype == dtype


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,F", [(1, 8), (3, 97), (70, 264), (2, 11008)])
def test_clamped_glu(dtype, T, F):
    x, b = rnd(5, T, 2 * F, scale=3.0).to(DEV, dtype), rnd(6, 2 * F).to(DEV)
    z = f64(x) + f64(b)
    close(ops.clamped_glu(x, b, 1.3), oracle.clamped_glu(z[:, :F], z[:, F:], 1.3), dtype)
    wide = rnd(7, T, 2 * F + 8).to(DEV, dtype)  # rows of a wider matrix
    z = f64(wide[:, :2 * F]) + f64(b)
    close(ops.clamped_glu(wide[:, :2 * F], b, 0.4), oracle.clamped_glu(z[:, :F], z[:, F:], 0.4), dtype)


@pytest.mark.parametrize("shape", [(1, 1), (3, 7), (5, 1024)])
def test_softcap(shape):
    z = rnd(8, *shape, scale=40.0).to(DEV)
    want = oracle.softcap(f64(z), 12.0)
    assert ops.softcap(z, 12.0) is not None
    close(z, want, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [64, 50])
def test_scaled_embedding(dtype, W):
    table = rnd(9, 20, W).to(DEV, dtype)
    sp = SpanBatch([[3, 19, 0]], [0], [0], DEV)
    want = f64(table)[[3, 19, 0]] * 0.3
    x, plain = ops.embed_rows(table, sp, scale=0.3, want_plain=True)
    close(x, want, torch.float32)
    close(plain, want, dtype)
    close(ops.embed_rows(table, sp), f64(table)[[3, 19, 0]], torch.float32)


# ---- the cache -----------------------------------------------------------------------------------------------------------

class Feeder:
    """Sequences in a latent cache: projections of every token are known in advance."""

    def __init__(self, dtype, q_rank, latent, rot, heads, window, scale=1.0, chunk=64, base=100.0, tokens=4096):
        self.dtype, self.q_rank, self.R, self.r, self.base = dtype, q_rank, latent, rot, base
        self.freq = None
        if rot:  # rounded, and what rounding left out
            f = torch.from_numpy(oracle.half_frequencies(rot, base))
            self.freq = torch.stack([f.float(), (f - f.float().double()).float()]).to(DEV)
        line = 128 // (2 if dtype == torch.bfloat16 else 4)
        mb = -(-(latent + rot) // line) * 128 * (tokens + 64 * chunk) / 2 ** 20
        self.cache = chunk_attn.Attention.latent(n_heads=heads, latent=latent, rotated=rot, scale=scale, window=window, chunk_size=chunk,
                                                 memory_mb=int(mb) + 1, dtype=dtype, device=DEV)
        self.q_norm, self.kv_norm = (1 + 0.2 * rnd(11, q_rank)).to(DEV), (1 + 0.2 * rnd(12, latent)).to(DEV)
        self.rows, self.n, self.proj, self.toks = [], {}, {}, {}

    def add(self, name, n, seed, toks=None, like=None):
        self.proj[name] = rnd(seed, n, self.q_rank + self.R + self.r, scale=2.0).to(DEV, self.dtype)
        self.toks[name] = toks if toks is not None else np.random.default_rng(seed).integers(0, 1 << 20, n).tolist()
        if like is not None:  # equal tokens have equal projections
            other, m = like
            self.proj[name][:m] = self.proj[other][:m]
            self.toks[name][:m] = self.toks[other][:m]

    def step(self, entries):
        """entries: [(name, tokens)].  Stores them; returns (spans, normalised query latents, row_entry or None)."""
        toks, starts, xs = [], [], []
        for name, k in entries:
            a = self.n.get(name, 0)
            toks.append(self.toks[name][a:a + k])
            starts.append(a)
            xs.append(self.proj[name][a:a + k])
        sp = SpanBatch(toks, starts, list(range(len(entries))), DEV)
        x = torch.cat(xs)
        names = [n for n, _ in entries]
        decode = self.cache.latent_decodes and names == self.rows and all(k == 1 for _, k in entries)
        if not decode:
            got = self.cache.extend([self.rows.index(n) if n in self.rows else -1 for n in names], toks)
            for n, r in zip(names, got):
                if n not in self.n:
                    self.rows.insert(r, n)
        c = self.cache.store_latent(x, sp.positions, self.q_norm, self.kv_norm, 0.1, self.freq, append_tokens=[t[0] for t in toks] if decode else None)
        for name, k in entries:
            self.n[name] = self.n.get(name, 0) + k
        return sp, c, None if decode else sp.entry_of

    def drop(self, name):
        row = self.rows.index(name)
        self.cache.remove_seq(row)
        del self.rows[row], self.n[name]

    def entries_of(self, name):
        """(latents, rotated key parts) the cache should hold, from the projections, in float64."""
        x = f64(self.proj[name])[:, self.q_rank:]
        c = oracle.plain_norm(x[:, :self.R], f64(self.kv_norm), 0.1)
        kr = oracle.rotate_halves(x[:, self.R:], np.arange(len(x)), self.r, self.base) if self.r else x[:, self.R:]
        return c, kr


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_rank,latent,rot", [(24, 64, 64), (30, 50, 6), (8, 128, 24), (1600, 512, 64), (7, 33, 2), (16, 48, 0)])
def test_stored_rows(dtype, q_rank, latent, rot):
    """What store_latent writes, read back through gather_latents: whole prompts, portions, decoded tokens, several rows, and
    chunks that were freed and are used again."""
    f = Feeder(dtype, q_rank, latent, rot, heads=2, window=0)
    everything = f.cache.reader(n_heads=1, scale=1.0, window=0)
    f.add("a", 200, 1)
    f.add("b", 90, 2)
    f.add("c", 140, 3, like=("a", 128))
    for entries in ([("a", 70)], [("b", 5), ("a", 2)], [("a", 1), ("b", 64)], [("c", 130)]):
        sp, c, _ = f.step(entries)
        x = torch.cat([f.proj[n][f.n[n] - k:f.n[n]] for n, k in entries])
        close(c, oracle.plain_norm(f64(x)[:, :q_rank], f64(f.q_norm), 0.1), dtype, "query latents")
        lat, kr = everything.gather_latents()
        want = [f.entries_of(n) for n, _ in entries]
        close(lat, np.concatenate([w[0][:f.n[n]] for w, (n, _) in zip(want, entries)]), dtype, "latents")
        close(kr[:, :rot] if rot else kr, np.concatenate([w[1][:f.n[n]] for w, (n, _) in zip(want, entries)]) if rot else np.zeros(kr.shape), dtype, "rotated")
        assert float(kr[:, rot:].abs().max()) == 0.0 if kr.shape[1] > rot else True
    for _ in range(9):  # decode steps, through the end of a chunk
        f.step([(n, 1) for n in f.rows])
    f.drop("b")
    f.add("d", 150, 4)
    f.step([("d", 3), ("a", 1)])
    f.step([("d", 147), ("a", 2)])
    lat, kr = everything.gather_latents()
    want = [f.entries_of(n)[0][:f.n[n]] for n in ("d", "a")]
    close(lat, np.concatenate(want), dtype, "latents in chunks used again")
    assert f.cache.device_status() == 0


def test_gathered_windows():
    """gather_latents brings exactly the rows the portions' windows touch."""
    f = Feeder(torch.bfloat16, 8, 64, 16, heads=2, window=70)
    f.add("a", 300, 1)
    f.add("b", 40, 2)
    f.step([("a", 250)])
    f.step([("b", 10), ("a", 20)])
    rows, pairs = f.cache.window_load()
    assert rows == 10 + 69 + 20 and pairs == 55 + 20 * 70
    lat, _ = f.cache.gather_latents()
    close(lat, np.concatenate([f.entries_of("b")[0][:10], f.entries_of("a")[0][181:270]]), torch.bfloat16)


# ---- attention -------------------------------------------------------------------------------------------------------------

def aimed(keys, n, heads, window, seed, scale):
    """Queries at positions 0 .. n-1 whose score is about 30 with the key at a distance that cycles through places just inside and
    outside the window, near ones, chunk borders and the first tokens, and small with the others.  keys [n, heads, d] float64."""
    g = np.random.default_rng(seed)
    d = keys.shape[2]
    q = g.standard_normal((n, heads, d)) / (scale * np.sqrt(d))
    dist = [window - 1, window, 0, 1, window + 1, window - 2, 63, 64, 65, 2, 127, 128, 10 ** 9, 10 ** 9 - 1]
    for i in range(n):
        for h in range(heads):
            t = dist[(i + 3 * h) % len(dist)]
            j = 10 ** 9 - t if t > 10 ** 8 else i - t  # the first two tokens, or t back
            if 0 <= j <= i:
                q[i, h] += 30.0 / scale * keys[j, h] / (keys[j, h] @ keys[j, h])
    return q


def turned_back(q, positions, dims, base):
    """The vector whose rotated last `dims` elements are those of q."""
    if dims == 0:
        return q
    return np.concatenate([q[..., :-dims], oracle.rotate_halves(q[..., -dims:], -np.asarray(positions), dims, base)], -1)



LATENT_CASES = {  # heads, latent, rot, window, chunk
    "small": (3, 24, 8, 20, 64),
    "odd": (5, 50, 6, 37, 64),
    "rows 16": (16, 128, 64, 64, 64),
    "rows 32": (30, 192, 16, 130, 64),
    "rows 64": (4, 512, 64, 65, 64),
    "more heads than a block": (72, 64, 64, 129, 64),
    "window of one": (7, 112, 24, 1, 64),
    "window beyond the sequence": (5, 130, 18, 5000, 64),
    "chunks of 16": (3, 64, 16, 33, 16),
    "wide latent": (2, 700, 64, 50, 64),
    "no window, no rotation": (4, 96, 0, 0, 64),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", sorted(LATENT_CASES))
def test_attention_in_the_latent_space(case, dtype):
    """Portions down to two tokens and decoding, two sequences of unequal length side by side, a sink per head."""
    heads, R, r, window, chunk = LATENT_CASES[case]
    if dtype == torch.float32 and heads > 16:
        heads = 9
    scale, n = 0.7, 200
    w = window or 10 ** 6
    f = Feeder(dtype, 8, R, r, heads, window, scale=scale, chunk=chunk)
    g = np.random.default_rng(3)
    sink = g.standard_normal(heads) * 4.0
    sink[0] = 14.0  # decides the sum for head 0
    sink_d = torch.from_numpy(sink).float().to(DEV)
    sink = f64(sink_d)
    f.add("a", n, 1)
    f.add("b", n - 23, 2)
    data = {}
    for name in ("a", "b"):
        c, kr = f.entries_of(name)
        # the values as stored: rounded to the cache's type
        c, kr = (f64(torch.from_numpy(t).to(dtype)) for t in (c, kr))
        keys = np.concatenate([c, kr], -1)[:, None].repeat(heads, 1)
        q = aimed(keys, len(c), heads, min(w, n), 7, scale)
        q = turned_back(q, np.arange(len(c)), r, f.base)
        qd = torch.from_numpy(q).to(dtype)
        qr = f64(qd)
        full = np.concatenate([qr[..., :R], oracle.rotate_halves(qr[..., R:], np.arange(len(c)), r, f.base)], -1) if r else qr
        want = oracle.windowed_attention(full, keys, c[:, None].repeat(heads, 1), scale, sink, w)
        data[name] = (qd.to(DEV), want, full, keys, c)
    if window and window < n:  # the aims have force: a window off by one, or a sink left out, would show
        qd, want, full, keys, c = data["a"]
        v = c[:, None].repeat(heads, 1)
        for other in (oracle.windowed_attention(full, keys, v, scale, sink, w + 1), oracle.windowed_attention(full, keys, v, scale, sink * 0 - 1e9, w)):
            assert np.abs(other - want).max() / np.abs(want).max() > 0.2
    got = {"a": [], "b": []}
    at = {"a": 0, "b": 0}
    plan = [[("a", 3)], [("b", 50), ("a", 2)], [("a", 70), ("b", 2)], [("b", 65)], [("a", 60), ("b", 1)], [("a", 2)]]
    plan += [None] * 40  # decode steps
    for entries in plan:
        entries = entries or [(x, 1) for x in f.rows]
        sp, _, row_entry = f.step(entries)
        q = torch.cat([data[x][0][at[x]:at[x] + k] for x, k in entries])
        out = f.cache.forward_latent(q[..., :R].contiguous(), q, sp.positions, f.freq, sink_d, row_entry)
        b = 0
        for x, k in entries:
            got[x].append(out[b:b + k])
            at[x] += k
            b += k
    for x in got:
        o = torch.cat(got[x])
        close(o, data[x][1][:len(o)], dtype, x)
    assert f.cache.device_status() == 0


EXPANDED_CASES = {  # heads, dim, rot, vdim, window
    "one panel each": (3, 64, 64, 64, 100),
    "large": (2, 128, 64, 128, 200),
    "odd panels": (5, 24, 8, 40, 33),
    "wide rotation": (2, 120, 128, 104, 64),
    "half panels": (3, 56, 24, 72, 1),
    "no window": (2, 72, 48, 128, 0),
}


@pytest.mark.parametrize("case", sorted(EXPANDED_CASES))
def test_attention_over_expanded_heads(case):
    """Prompts and portions behind a context, several per step, blocks of one token up to several blocks, a sink per head."""
    heads, dim, r, vdim, window = EXPANDED_CASES[case]
    dtype, R, scale, w = torch.bfloat16, 64, 0.6, window or 10 ** 6
    f = Feeder(dtype, 8, R, r, heads, window, scale=scale)
    assert f.cache.latent_expands(dim, vdim) and not f.cache.latent_expands(dim + 1, vdim) and not f.cache.latent_expands(136, vdim)
    g = np.random.default_rng(4)
    sink_d = torch.from_numpy(np.concatenate([[13.0], g.standard_normal(heads - 1) * 4.0])).float().to(DEV)
    sink = f64(sink_d)
    w_ukv = rnd(6, heads * (dim + vdim), R, scale=R ** -0.5).to(DEV, dtype)
    lens = {"a": 700, "b": 300, "c": 1, "d": 257}
    data = {}
    for k, (name, n) in enumerate(lens.items()):
        f.add(name, n, 20 + k)
        c, kr = (f64(torch.from_numpy(t).to(dtype)) for t in f.entries_of(name))
        kv = f64(torch.from_numpy(c).to(DEV, dtype) @ w_ukv.t())
        keys = np.concatenate([kv[:, :heads * dim].reshape(n, heads, dim), kr[:, None].repeat(heads, 1)], -1)
        vals = kv[:, heads * dim:].reshape(n, heads, vdim)
        q = torch.from_numpy(turned_back(aimed(keys, n, heads, min(w, n), 8, scale), np.arange(n), r, f.base)).to(dtype)
        full = np.concatenate([f64(q)[..., :dim], oracle.rotate_halves(f64(q)[..., dim:], np.arange(n), r, f.base)], -1)
        data[name] = (q.to(DEV), oracle.windowed_attention(full, keys, vals, scale, sink, w))
        if name == "b" and window:  # the aims have force
            for other in (oracle.windowed_attention(full, keys, vals, scale, sink, w + 1), oracle.windowed_attention(full, keys, vals, scale, sink * 0 - 1e9, w)):
                d = np.abs(other - data[name][1]) / np.abs(data[name][1]).max()
                assert d.max() > 0.2 and np.sqrt((d ** 2).mean()) > 1.5e-2
    at = dict.fromkeys(lens, 0)
    for entries in ([("a", 300)], [("b", 128), ("a", 2), ("c", 1)], [("a", 64), ("d", 257), ("b", 130)], [("b", 42), ("a", 334)]):
        sp, _, _ = f.step(entries)
        lat, rot = f.cache.gather_latents()
        q = torch.cat([data[x][0][at[x]:at[x] + k] for x, k in entries]).contiguous()
        out = f.cache.forward_expanded(q, lat @ w_ukv.t(), rot, sp.positions, f.freq, sink_d, vdim)
        b = 0
        for x, k in entries:
            # the latents the oracle starts from are rounded after another order of operations: a few differ by one step
            want = data[x][1][at[x]:at[x] + k]
            err = np.abs(f64(out[b:b + k]) - want) / np.abs(want).max()
            assert err.max() < 0.1 and np.sqrt((err ** 2).mean()) < 4e-3, (x, err.max(), np.sqrt((err ** 2).mean()))
            at[x] += k
            b += k
    assert f.cache.device_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_readers(dtype):
    """Layers that read one cache with other heads, scales and windows, in portions and in decode steps over a shared prefix,
    while rows come and go; a reader refuses to change what it reads."""
    R, r, n = 96, 16, 260
    f = Feeder(dtype, 8, R, r, heads=4, window=50, scale=0.5)
    views = {"owner": (f.cache, 4, 0.5, 50)}
    for heads, scale, window in ((4, 0.5, 50), (4, 0.5, 50), (7, 0.9, 131), (20, 0.3, 1)):
        sibling = views["r0"][0] if len(views) == 2 else None
        views["r%d" % (len(views) - 1)] = (f.cache.reader(n_heads=heads, scale=scale, window=window, sibling=sibling), heads, scale, window)
    f.add("a", n, 1)
    f.add("b", n, 2, like=("a", 130))
    f.add("c", n, 3, like=("a", 70))
    f.add("d", n, 4)
    sinks = {v: torch.linspace(-1, 3, x[1], device=DEV) for v, x in views.items()}

    def check(entries):
        starts = {x: f.n.get(x, 0) for x, _ in entries}
        sp, _, row_entry = f.step(entries)
        for v, (view, heads, scale, window) in views.items():
            q, want = [], []
            for x, k in entries:
                c, kr = (f64(torch.from_numpy(t).to(dtype))[:starts[x] + k] for t in f.entries_of(x))
                keys = np.concatenate([c, kr], -1)[:, None].repeat(heads, 1)
                qq = torch.from_numpy(turned_back(aimed(keys, len(c), heads, window, 9, scale), np.arange(len(c)), r, f.base)).to(dtype)
                full = np.concatenate([f64(qq)[..., :R], oracle.rotate_halves(f64(qq)[..., R:], np.arange(len(c)), r, f.base)], -1)
                # only the step's rows are wanted
                part = np.zeros((k, heads, R))
                for i in range(starts[x], starts[x] + k):
                    seen = list(oracle.window_positions(i, window))
                    for h in range(heads):
                        part[i - starts[x], h] = oracle.sink_softmax(keys[seen, h] @ full[i, h] * scale, f64(sinks[v])[h]) @ c[seen]
                q.append(qq[starts[x]:])
                want.append(part)
            q = torch.cat(q).to(DEV)
            out = view.forward_latent(q[..., :R].contiguous(), q, sp.positions, f.freq, sinks[v], row_entry)
            close(out, np.concatenate(want), dtype, v)

    check([("a", 140)])
    check([("b", 135), ("c", 70)])
    for _ in range(3):
        check([(x, 1) for x in f.rows])
    f.drop("b")
    check([(x, 1) for x in f.rows])
    check([("d", 62)])
    for _ in range(3):
        check([(x, 1) for x in f.rows])
    reader = views["r1"][0]
    for call in (lambda: reader.remove_seq(0), lambda: reader.extend([0], [[1]]), lambda: reader.clear(), lambda: reader.reserve()):
        with pytest.raises(RuntimeError, match="reader"):
            call()
    with pytest.raises(RuntimeError, match="separate keys"):
        f.cache.add_seq(tokens=[1], k=torch.zeros(1, 1, R + r, device=DEV), v=torch.zeros(1, 1, R, device=DEV))
    assert all(v[0].device_status() == 0 for v in views.values())


def test_angles_far_from_the_start():
    """In fp32 the rotation at position 100 000 is as exact as at the start: angles are not rounded to one fp32 number."""
    f = Feeder(torch.float32, 8, 32, 16, heads=1, window=0, base=3.0, tokens=128)
    x = rnd(3, 1, 8 + 32 + 16).to(DEV)
    pos = 100_000
    sp = SpanBatch([[1]], [pos], [0], DEV)
    f.cache.extend([-1], [[1]])
    f.cache.store_latent(x, sp.positions, f.q_norm, f.kv_norm, 0.1, f.freq)
    _, kr = f.cache.gather_latents()
    close(kr[:, :16], oracle.rotate_halves(f64(x)[:, 40:], [pos], 16, 3.0), torch.float32)
