"""Plain CPU oracle of the Bikelix decoder: one function per mechanism, one sequence at a time, every key visited
by a loop over positions, numpy in float64.  Shares no code with the product and knows nothing of caches, chunks,
batches or of the product's way to fold projections.

`weights` maps tensor names to arrays; `cfg` is the parsed config.json.
"""
import numpy as np


def root_mean_square(x, eps):
    return np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def plain_norm(x, w, eps):
    """RMS norm whose weight is stored as it is applied."""
    return x / root_mean_square(x, eps) * w


def centred_norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return x / root_mean_square(x, eps) * (1.0 + w)


def half_frequencies(dims, base):
    return base ** (-2.0 * np.arange(dims // 2) / dims)


def rotate_halves(x, positions, dims, base):
    """x [T, ..., d]: element i and element i + dims / 2 of the leading `dims` turned by position * frequency i."""
    half = dims // 2
    a = np.asarray(positions, np.float64)[:, None] * half_frequencies(dims, base)
    a = a.reshape((a.shape[0],) + (1,) * (x.ndim - 2) + (half,))
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), x[..., dims:]], -1)


def window_positions(i, size):
    """The positions that position i sees."""
    return range(max(0, i - size + 1), i + 1)


def sink_softmax(scores, sink):
    """Weights of the scored entries when one more entry of score `sink` takes part and is then dropped."""
    m = max(scores.max(), sink)
    e = np.exp(scores - m)
    return e / (e.sum() + np.exp(sink - m))


def windowed_attention(q, k, v, scale, sink, size):
    """q, k [T, H, d], v [T, H, dv], sink [H]."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        seen = list(window_positions(i, size))
        for h in range(H):
            p = sink_softmax(k[seen, h] @ q[i, h] * scale, sink[h])
            out[i, h] = p @ v[seen, h]
    return out


def query_heads(x, w, p, m, eps):
    """[T, heads, dim + rot_dim], the last part turned."""
    T, H, d, r = x.shape[0], m["heads"], m["dim"], m["rot_dim"]
    c = plain_norm(x @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (c @ w[p + "uq"].T).reshape(T, H, d + r)
    turned = rotate_halves(q[..., d:], np.arange(T), m["rot"]["dims"], m["rot"]["base"])
    return np.concatenate([q[..., :d], turned], -1)


def latent_entries(x, w, p, m, eps):
    """What a layer keeps of every token: the latent [T, kv_rank] and the key part all heads share [T, rot_dim], turned."""
    R = m["kv_rank"]
    kv = x @ w[p + "dkv"].T
    c = plain_norm(kv[:, :R], w[p + "dkv.norm"], eps)
    return c, rotate_halves(kv[:, R:], np.arange(x.shape[0]), m["rot"]["dims"], m["rot"]["base"])


def latent_attention(x, w, p, m, eps, entries):
    """entries: (latent, shared key part) of the layer that owns the cache read here."""
    T, H, d, r, dv = x.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, shared = entries
    q = query_heads(x, w, p, m, eps)
    k = (c @ w[p + "uk"].T).reshape(T, H, d)
    k = np.concatenate([k, np.broadcast_to(shared[:, None], (T, H, r))], -1)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    o = windowed_attention(q, k, v, m["scale"], w[p + "sink"], m["mask"]["size"])
    return o.reshape(T, H * dv) @ w[p + "o"].T


def clamped_glu(gate, up, limit):
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0)


def dense_ff(x, w, p, limit):
    gate = x @ w[p + "gate"].T + w[p + "gate.b"]
    up = x @ w[p + "up"].T + w[p + "up.b"]
    return clamped_glu(gate, up, limit) @ w[p + "down"].T + w[p + "down.b"]


def softcap(z, cap):
    return cap * np.tanh(z / cap)


def forward(tokens, w, cfg):
    """Returns (logits [T, vocab], [residual stream after each layer])."""
    w = {k: np.asarray(v, np.float64) for k, v in w.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    after, kept = [], {}
    for i, spec in enumerate(cfg["layers"]):
        if spec["type"] != "latent_attention":
            raise ValueError(spec["type"])
        p, m = "l%d." % i, spec["mixer"]
        owner = m.get("kv_from")
        if owner is None:
            owner = i
            kept[i] = latent_entries(x, w, p + "mix.", m, eps)
        r = latent_attention(x, w, p + "mix.", m, eps, kept[owner])
        x = centred_norm(alpha * x + r, w[p + "norm1"], eps)
        if spec["mlp"] is not None:
            r = dense_ff(x, w, p + "mlp.", spec["mlp"]["limit"])
            x = centred_norm(alpha * x + r, w[p + "norm2"], eps)
        after.append(x)
    logits = centred_norm(x, w["final.norm"], eps) @ w["embed"].T
    return softcap(logits, cfg["logit_softcap"]), after
