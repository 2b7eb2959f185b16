"""The block kernels one by one against the plain oracle: spans of several lengths, states carried between steps, slots
used again, sizes that are no multiple of a vector."""
import numpy as np
import pytest
import torch

import chunk_attn
import gagorax_oracle as oracle
from chunk_attn import SpanBatch, ops

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")
DTYPES = [torch.float32, torch.bfloat16]
EPS = {torch.float32: 2e-5, torch.bfloat16: 1.6e-2}


def rnd(seed, *shape, scale=1.0):
    return torch.from_numpy(np.random.default_rng(seed).standard_normal(shape).astype(np.float32) * scale)


def close(got, want, dtype, what=""):
    want = np.asarray(want, np.float64)
    err = np.abs(got.double().cpu().numpy() - want).max()
    assert err <= EPS[dtype] * max(1.0, np.abs(want).max()), "%s: %g" % (what, err)


def plan(lens_per_step, slots):
    """Spans of a schedule: step s brings lens_per_step[s][e] tokens of sequence e (0: it rests)."""
    at = [0] * len(slots)
    for lens in lens_per_step:
        live = [e for e, n in enumerate(lens) if n]
        yield [(e, at[e], lens[e]) for e in live], SpanBatch([[0] * lens[e] for e in live], [at[e] for e in live],
                                                             [slots[e] for e in live], DEV)
        for e in live:
            at[e] += lens[e]


SCHEDULES = [[[5, 1, 130]], [[1, 1, 1]] * 6, [[2, 64, 3], [0, 1, 65], [70, 2, 0], [1, 1, 1]], [[200, 0, 63], [1, 3, 1], [2, 129, 64]]]


def run(schedule, inputs, step):
    """Feeds the rows of `inputs` ([T, ...] per sequence) through step(rows, spans) and returns the outputs per sequence."""
    out = [[] for _ in inputs]
    for entries, spans in plan(schedule, slots=[4, 0, 2]):
        rows = torch.cat([inputs[e][a:a + n] for e, a, n in entries])
        y = step(rows, spans)
        base = 0
        for e, _, n in entries:
            out[e].append(y[base:base + n])
            base += n
    return [torch.cat(o) if o else None for o in out]


def lengths(schedule):
    return [sum(l[e] for l in schedule) for e in range(3)]


@pytest.mark.parametrize("schedule", SCHEDULES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 97])
def test_token_shift(width, dtype, schedule):
    mu = rnd(1, width).to(DEV)
    state = torch.full((5, width), 7.0, device=DEV)  # stale: ignored at position 0
    xs = [rnd(10 + e, n, width) for e, n in enumerate(lengths(schedule))]
    out = run(schedule, xs, lambda rows, sp: torch.stack(ops.token_shift(rows.to(DEV), mu, state, sp, dtype), 1))
    for x, y in zip(xs, out):
        close(y[:, 0], x.numpy(), dtype)
        close(y[:, 1], oracle.token_shift(x.double().numpy(), mu.cpu().double().numpy()), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 97, 4096, 9000])
def test_gated_norm_add(width, dtype):
    T, eps = 5, 1e-3
    x, r, gate = rnd(1, T, width), rnd(2, T, width).to(dtype), rnd(3, T, 2 * width).to(dtype)[:, width:]
    b, w = rnd(4, width), rnd(5, width)
    got = x.clone().to(DEV)
    gate_dev = torch.zeros(T, 2 * width, dtype=dtype, device=DEV)
    gate_dev[:, width:] = gate.to(DEV)
    plain, shifted = ops.gated_norm_add(got, r.to(DEV), gate_dev[:, width:], b.to(DEV), w.to(DEV), eps)
    g = r.double().numpy() * oracle.sigmoid(gate.double().numpy() + b.double().numpy())
    want = x.double().numpy() + oracle.rms_norm(g, w.double().numpy(), eps)
    close(got, want, torch.float32)
    close(plain, want, dtype)
    assert shifted is None
    # with the next layer's token shift: the first token of slot 1, a later one of slot 0 ...
    mu, state = rnd(6, width), rnd(7, T, width)
    sp = SpanBatch([[0]] * T, [3, 0, 1, 9, 0], [0, 1, 4, 3, 2], DEV)
    got2, st = x.clone().to(DEV), state.clone().to(DEV)
    plain2, shifted = ops.gated_norm_add(got2, r.to(DEV), gate_dev[:, width:], b.to(DEV), w.to(DEV), eps, next_mu=mu.to(DEV),
                                         next_state=st, spans=sp)
    assert torch.equal(got, got2) and torch.equal(plain, plain2)
    for t, (start, slot) in enumerate(zip([3, 0, 1, 9, 0], [0, 1, 4, 3, 2])):
        prev = state[slot].double().numpy() if start else 0.0
        close(shifted[t], want[t] + (prev - want[t]) * mu.double().numpy(), dtype)
        close(st[slot], want[t], torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 97])
def test_norms_and_gelu(width, dtype):
    x, w, gate = rnd(1, 6, width), rnd(2, width), rnd(3, 4, width).to(dtype)
    rows = torch.tensor([5, 0, 0, 3], dtype=torch.int32, device=DEV)
    y = ops.norm_rows(x.to(DEV), w.to(DEV), 1e-2, dtype, rows=rows, gate=gate.to(DEV))
    want = oracle.rms_norm(x.double().numpy(), w.double().numpy(), 1e-2)[[5, 0, 0, 3]] * oracle.sigmoid(gate.double().numpy())
    close(y, want, dtype)
    z = (rnd(4, 7, 2 * width) * 3).to(dtype)
    close(ops.gelu_tanh(z.to(DEV)[:, :width]), oracle.gelu_tanh(z[:, :width].double().numpy()), dtype)


@pytest.mark.parametrize("schedule", SCHEDULES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channels,taps", [(64, 4), (33, 2), (130, 1), (64, 3), (48, 7)])
def test_convolution(channels, taps, dtype, schedule):
    f, b = rnd(1, channels, taps), rnd(2, channels)
    state = torch.full((5, taps - 1, channels), 7.0, device=DEV)
    xs = [rnd(10 + e, n, channels).to(dtype) for e, n in enumerate(lengths(schedule))]
    wide = lambda rows: torch.cat([rows, rows], 1).to(DEV)[:, :channels]  # a slice of wider rows
    out = run(schedule, xs, lambda rows, sp: ops.conv_silu(wide(rows), f.to(DEV), b.to(DEV), state, sp))
    for x, y in zip(xs, out):
        close(y, oracle.silu(oracle.causal_conv(x.double().numpy(), f.double().numpy(), b.double().numpy())), dtype)


@pytest.mark.parametrize("schedule", SCHEDULES + [[[700, 0, 129], [333, 3, 1]]])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channels,states", [(64, 16), (33, 5), (130, 40), (40, 1), (128, 64), (24, 100)])
def test_selective_scan(channels, states, dtype, schedule):
    lens = lengths(schedule)
    A, D, bias = -torch.exp(rnd(1, channels, states)), rnd(2, channels), rnd(3, channels) - 2
    state = torch.full((5, channels, states), 7.0, device=DEV)
    x = [rnd(10 + e, n, channels).to(dtype).float() for e, n in enumerate(lens)]
    z = [rnd(20 + e, n, channels).to(dtype).float() for e, n in enumerate(lens)]
    dt = [rnd(30 + e, n, channels) for e, n in enumerate(lens)]
    bc = [rnd(40 + e, n, 2 * states) for e, n in enumerate(lens)]
    packed = [torch.cat(p, 1) for p in zip(x, z, dt, bc)]

    def step(rows, sp):
        rows = rows.to(DEV)
        a, b, c, d = rows.split([channels, channels, channels, 2 * states], 1)
        return ops.selective_scan(a.to(dtype).contiguous(), b.to(dtype), c.contiguous(), bias.to(DEV), A.to(DEV), d, D.to(DEV), state, sp)

    out = run(schedule, packed, step)
    for e in range(3):
        n = lambda t: t.double().numpy()
        y, S = oracle.selective_scan(n(x[e]), oracle.softplus(n(dt[e]) + n(bias)), n(A), n(bc[e])[:, :states], n(bc[e])[:, states:], n(D))
        close(out[e], y * oracle.silu(n(z[e])), dtype)
        if lens[e]:
            close(state[[4, 0, 2][e]], S, torch.float32, "state")


@pytest.mark.parametrize("schedule", SCHEDULES + [[[700, 0, 129], [333, 3, 1]]])  # the last one takes runs of blocks in two passes
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dk,dv,decay", [(16, 16, [0.9, 0.5]), (20, 36, [1.0]), (64, 64, [0.999, 0.0, 0.7]), (128, 128, [0.98, 0.9999]),
                                         (128, 64, [0.99]), (48, 80, [0.95, 0.3])])
def test_decay_attention(dk, dv, decay, dtype, schedule):
    lens, H = lengths(schedule), len(decay)
    state = torch.full((5, H, dk, dv), 7.0, device=DEV)
    d = torch.tensor(decay, device=DEV)
    xs = [(rnd(10 + e, n, H * (2 * dk + dv) + 8)).to(dtype) for e, n in enumerate(lens)]
    out = run(schedule, xs, lambda rows, sp: ops.decay_attention(rows.to(DEV), d, dk, dv, state, sp))
    for e in range(3):
        if not lens[e]:
            continue
        a = oracle.silu(xs[e].double().numpy())
        q, k, v = (m.reshape(lens[e], H, -1) for m in np.split(a[:, :H * (2 * dk + dv)], [H * dk, 2 * H * dk], 1))
        o, S = oracle.decayed_linear_attention(q, k, v, decay)
        close(out[e], o.reshape(lens[e], -1), dtype)
        close(state[[4, 0, 2][e]], S, torch.float32 if dtype == torch.float32 else torch.bfloat16, "state")


# ---- attention with a head shape --------------------------------------------------------------------------------------
SHAPES = [(4, 2, 40, 24, 24), (2, 2, 128, 128, 128), (8, 1, 64, 64, 16), (3, 3, 20, 36, 20), (6, 2, 256, 256, 64), (4, 4, 64, 128, 64),
          (16, 2, 128, 64, 0), (5, 1, 72, 8, 2)]


def oracle_attention(x, shape, qn, kn, eps, base, scale, sink=True):
    H, G, dk, dv, rot = shape
    T = x.shape[0]
    q, k, v = np.split(x, [H * dk, (H + G) * dk], 1)
    pos = np.arange(T)
    q = oracle.rotary(oracle.rms_norm(q.reshape(T, H, dk), qn, eps), pos, rot, base)
    k = oracle.rotary(oracle.rms_norm(k.reshape(T, G, dk), kn, eps), pos, rot, base)
    v = oracle.rotary(v.reshape(T, G, dv), pos, dv, base)
    return oracle.rotary(oracle.sink_attention(q, k, v, scale), -pos, dv, base)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("chunk", [64, 16])
def test_attention_over_the_chunk_pool(shape, dtype, chunk):
    """Norm, rotations, sink, groups and the walk over chunks: prompts, portions, decoding of several rows, a shared
    prefix, and rows that leave."""
    H, G, dk, dv, rot = shape
    eps, base, scale = 1e-4, 1000.0, 1.7 * dk ** -0.5
    cache = chunk_attn.Attention.shaped(n_heads=H, n_kv_heads=G, d_key=dk, d_value=dv, scale=scale, sink=True, chunk_size=chunk,
                                        memory_mb=64, dtype=dtype, device=DEV)
    qn, kn = rnd(1, dk) * 0.2 + 1, rnd(2, dk) * 0.2 + 1
    freq = lambda n: torch.from_numpy(oracle.pair_frequencies(n, base).astype(np.float32)).to(DEV)
    kf, vf = freq(rot) if rot else None, freq(dv)
    width = (H + G) * dk + G * dv
    lens = [150, 133, 70, 1]
    xs = [rnd(10 + e, n + 40, width).to(dtype) for e, n in enumerate(lens)]
    ids = [[1000 * e + t for t in range(n + 40)] for e, n in enumerate(lens)]
    xs[1][:130] = xs[0][:130]  # the same tokens, and therefore the same projections
    ids[1][:130] = ids[0][:130]
    want = [oracle_attention(x.double().numpy(), shape, qn.double().numpy(), kn.double().numpy(), eps, base, scale) for x in xs]
    at, order, got = [0] * 4, [], [[] for _ in lens]

    def feed(entries):
        """entries: [(request, tokens)]"""
        decode = [e for e, _ in entries] == order and all(n == 1 for _, n in entries)
        rows = [order.index(e) if e in order else -1 for e, _ in entries]
        toks = [ids[e][at[e]:at[e] + n] for e, n in entries]
        if not decode:
            for (e, _), was, r in zip(entries, rows, cache.extend(rows, toks)):
                if was < 0:
                    order.insert(r, e)
        sp = SpanBatch(toks, [at[e] for e, _ in entries], [e for e, _ in entries], DEV)
        x = torch.cat([xs[e][at[e]:at[e] + n] for e, n in entries]).to(DEV)
        q = cache.store_qkv(x, sp.positions, qn.to(DEV), kn.to(DEV), eps, rot, kf, vf, append_tokens=[t[0] for t in toks] if decode else None)
        o = cache.forward_rows(q, sp.positions, vf, None if decode else sp.entry_of)
        base_ = 0
        for e, n in entries:
            got[e].append(o[base_:base_ + n])
            base_ += n
            at[e] += n

    feed([(0, 150)])
    feed([(1, 2), (2, 64), (3, 1)])
    feed([(2, 6)])
    feed([(1, 131), (0, 1)])
    for _ in range(20):
        feed([(e, 1) for e in order])
    cache.remove_seq(order.index(2))
    order.remove(2)
    for _ in range(18):
        feed([(e, 1) for e in order])
    for e in range(4):
        o = torch.cat(got[e])
        close(o, want[e][:o.shape[0]], dtype, "request %d" % e)
    assert cache.device_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_sink_and_large_scores(dtype):
    """One token: the output is v e^s / (1 + e^s).  Scores far below 0 leave everything to the sink, far above nothing."""
    for scale in (0.0, 1.0, -3.0, 30.0, -30.0):
        cache = chunk_attn.Attention.shaped(n_heads=2, n_kv_heads=1, d_key=16, d_value=16, scale=scale, sink=True, chunk_size=8,
                                            memory_mb=4, dtype=dtype, device=DEV)
        x = torch.ones(1, 64)  # q = k = 1: q . k = 16
        x[0, 48:] = torch.arange(16.0)
        sp = SpanBatch([[3]], [0], [0], DEV)
        cache.extend([-1], [[3]])
        q = cache.store_qkv(x.to(DEV, dtype), sp.positions)
        o = cache.forward_rows(q, sp.positions, None, sp.entry_of)
        close(o[0, 1], np.arange(16.0) / (1 + np.exp(-16.0 * scale)), dtype)
        # without the unit term the one token takes all
        plain = chunk_attn.Attention.shaped(n_heads=2, n_kv_heads=1, d_key=16, d_value=16, scale=scale, chunk_size=8, memory_mb=4,
                                            dtype=dtype, device=DEV)
        plain.extend([-1], [[3]])
        o = plain.forward_rows(plain.store_qkv(x.to(DEV, dtype), sp.positions), sp.positions, None, sp.entry_of)
        close(o[0, 0], np.arange(16.0), dtype)


def test_shaped_cache_takes_plain_kv_too():
    """add_seq / append_token with ready keys and values (padded inside), then forward_rows."""
    g = torch.Generator().manual_seed(3)
    cache = chunk_attn.Attention.shaped(n_heads=4, n_kv_heads=2, d_key=20, d_value=12, scale=0.3, chunk_size=16, memory_mb=8,
                                        dtype=torch.float32, device=DEV)
    k, v = torch.randn(41, 2, 20, generator=g), torch.randn(41, 2, 12, generator=g)
    cache.add_seq(tokens=list(range(40)), k=k[:40].to(DEV), v=v[:40].to(DEV))
    cache.append_token(tokens=[40], k=k[40:].to(DEV), v=v[40:].to(DEV))
    q = torch.randn(1, 4, 20, generator=g)
    o = cache.forward_rows(q.to(DEV), torch.tensor([40], dtype=torch.int32, device=DEV))
    s = torch.einsum("hd,thd->ht", q[0], k.repeat_interleave(2, 1)) * 0.3
    want = torch.einsum("ht,thd->hd", s.softmax(-1), v.repeat_interleave(2, 1))
    close(o[0], want.numpy(), torch.float32)
