"""Plain CPU oracle of the Gagorax decoder: one function per mechanism, one sequence at a time, one
token at a time wherever a state is involved, numpy in float64.  Shares no code with the product and
knows nothing of caches, chunks, slots or batches.

`weights` maps tensor names to arrays; `cfg` is the parsed config.json.
"""
import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def token_shift(h, mu):
    """h [T, width]: each token mixed with the one before it (zeros before the first)."""
    prev = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    return h + (prev - h) * mu


def rotate_pairs(x, angle):
    """x [..., dims] as interleaved pairs (2i, 2i + 1), pair i turned by angle[..., i]."""
    u, v = x[..., 0::2], x[..., 1::2]
    c, s = np.cos(angle), np.sin(angle)
    out = np.empty_like(x)
    out[..., 0::2] = u * c - v * s
    out[..., 1::2] = v * c + u * s
    return out


def pair_frequencies(dims, base):
    return base ** (-2.0 * np.arange(dims // 2) / dims)


def rotary(x, positions, dims, base):
    """x [T, heads, d]: the first `dims` dimensions of every head turned by the token's position."""
    a = np.asarray(positions, np.float64)[:, None, None] * pair_frequencies(dims, base)
    return np.concatenate([rotate_pairs(x[..., :dims], np.broadcast_to(a, x.shape[:2] + (dims // 2,))), x[..., dims:]], -1)


def sink_attention(q, k, v, scale):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv]; causal; one added to the softmax's denominator."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        for h in range(H):
            s = k[:i + 1, h // per] @ q[i, h] * scale
            m = max(s.max(), 0.0)
            e = np.exp(s - m)
            out[i, h] = e @ v[:i + 1, h // per] / (np.exp(-m) + e.sum())
    return out


def attention_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(T)
    q = rms_norm((h @ w[p + "q"].T).reshape(T, H, dk), w[p + "q.norm"], eps)
    k = rms_norm((h @ w[p + "k"].T).reshape(T, G, dk), w[p + "k.norm"], eps)
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    q, k = rotary(q, pos, dims, base), rotary(k, pos, dims, base)
    v = rotary(v, pos, dv, base)
    o = sink_attention(q, k, v, m["scale"])
    o = rotary(o, -pos, dv, base)
    return o.reshape(T, H * dv) @ w[p + "o"].T


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, K]: per channel, the last tap is the current token's."""
    K = taps.shape[1]
    xp = np.concatenate([np.zeros((K - 1, x.shape[1])), x])
    return sum(xp[j:j + x.shape[0]] * taps[:, j] for j in range(K)) + bias


def selective_scan(x, dt, A, B, C, D, state=None):
    """x, dt [T, C]; A [C, N]; B, C [T, N]; returns (y [T, C], final state [C, N])."""
    S = np.zeros_like(A) if state is None else state.copy()
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def mamba_mixer(h, w, p, m):
    n, r = m["state"], m["dt_rank"]
    x, z = np.split(h @ w[p + "in"].T, 2, axis=-1)
    x = silu(causal_conv(x, w[p + "conv"], w[p + "conv.b"]))
    proj = x @ w[p + "x"].T
    dt = softplus(proj[:, :r] @ w[p + "dt"].T + w[p + "dt.b"])
    y, _ = selective_scan(x, dt, -np.exp(w[p + "A_log"]), proj[:, r:r + n], proj[:, r + n:], w[p + "D"])
    return (y * silu(z)) @ w[p + "o"].T


def decayed_linear_attention(q, k, v, decay, state=None):
    """q, k [T, H, dk], v [T, H, dv]: S <- decay S + k v^T, o = S^T q; returns (o, final S)."""
    S = np.zeros((q.shape[1], q.shape[2], v.shape[2])) if state is None else state.copy()
    o = np.zeros(v.shape)
    for t in range(q.shape[0]):
        S = np.asarray(decay)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hkv,hk->hv", S, q[t])
    return o, S


def lightning_mixer(h, w, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q = silu(h @ w[p + "q"].T).reshape(T, H, m["dim"])
    k = silu(h @ w[p + "k"].T).reshape(T, H, m["dim"])
    v = silu(h @ w[p + "v"].T).reshape(T, H, m["vdim"])
    o, _ = decayed_linear_attention(q, k, v, m["decay"])
    o = rms_norm(o.reshape(T, -1), w[p + "norm"], eps) * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def dense_ff(h, w, p):
    return gelu_tanh(h @ w[p + "up"].T) @ w[p + "down"].T


def layer(x, w, i, spec, eps):
    p = "l%d." % i
    h = token_shift(x, w[p + "shift"])
    kind, m = spec["type"], spec["mixer"]
    if kind == "mamba1":
        r = mamba_mixer(h, w, p + "mix.", m)
    elif kind == "attention":
        r = attention_mixer(h, w, p + "mix.", m, eps)
    elif kind == "lightning":
        r = lightning_mixer(h, w, p + "mix.", m, eps)
    else:
        raise ValueError(kind)
    x = x + rms_norm(r * sigmoid(x @ w[p + "rg1"].T + w[p + "rg1.b"]), w[p + "norm1"], eps)
    if spec["mlp"] is not None:
        r = dense_ff(x, w, p + "mlp.")
        x = x + rms_norm(r * sigmoid(x @ w[p + "rg2"].T + w[p + "rg2.b"]), w[p + "norm2"], eps)
    return x


def forward(tokens, w, cfg):
    """Returns (logits [T, vocab], [residual stream after each layer])."""
    w = {k: np.asarray(v, np.float64) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    after = []
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, w, i, spec, eps)
        after.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"], after
