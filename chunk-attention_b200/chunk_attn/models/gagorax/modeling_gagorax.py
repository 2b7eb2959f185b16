"""Gagorax: a decoder of Mamba, rotary attention and linear-attention layers over one fp32 residual stream.

A layer is x += norm(gate * mixer(shift(x))) and, when it has a feed-forward, x += norm(gate * ff(x)): the sublayers
read the stream itself, the RMS norm is on their output.  Tensors are named `embed`, `l<i>.norm1`, `l<i>.shift`,
`l<i>.rg1`, `l<i>.mix.*`, `l<i>.mlp.*`, ..., `final.norm`, `head`.

The model runs STEPS.  A step brings the next tokens of any number of sequences (a whole prompt, a portion of one, a
decoded token), laid end to end; everything older comes from the caches: one `chunk_attn.Attention` per attention
layer, one `RecurrentState` for the rest (shifted rows, convolution windows, scan and linear-attention states).
Prefill, decode and continued portions are the same code; a step of one token for every row takes the decode kernels,
which walk shared prefixes once.  Call protocol as the other decoder: `model(seqs, kv_caches, prefill)` returns the
next token of each sequence, `model.create_kv_caches()` makes the caches, so `ModelHost` serves it unchanged.

Per sublayer: projections are library GEMMs with their weights concatenated where they read the same rows; everything
between them is a kernel of `chunk_attn.ops` or of the cache, with fp32 arithmetic on the residual, norms, angles,
scores, gates, step sizes and states.
"""
import math

import torch
from torch.nn.functional import linear

import chunk_attn
from chunk_attn import SpanBatch, ops

from ..recurrent_state import RecurrentState
from .configuration_gagorax import GagoraxConfig


def linear_f32(x, w):
    """x W^T with the fp32 accumulator as the result."""
    if x.dtype == torch.float32:
        return linear(x, w)
    return torch.mm(x, w.t(), out_dtype=torch.float32)


def pair_frequencies(dims, base, device):
    """Radians per position of the dims / 2 rotation pairs, rounded once to fp32."""
    f = float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    return f.to(torch.float32).to(device)


class Weights:
    """The named tensors of a model, placed on the device: matrices in the model's dtype, vectors in fp32."""

    def __init__(self, tensors, config):
        self.tensors, self.config = tensors, config

    def matrix(self, *names):
        """One matrix, or several that read the same input, stacked."""
        ws = [self.tensors[n].to(device=self.config.torch_device, dtype=self.config.torch_dtype) for n in names]
        return (ws[0] if len(ws) == 1 else torch.cat(ws)).contiguous()

    def vector(self, name):
        return self.tensors[name].to(device=self.config.torch_device, dtype=torch.float32).contiguous()


class MambaMixer:
    def __init__(self, w, p, m, config, key):
        self.inner, self.n_states, self.rank, self.key = m["inner"], m["state"], m["dt_rank"], key
        self.taps_n = m["conv"]
        self.w_in, self.w_x, self.w_dt, self.w_o = (w.matrix(p + n) for n in ("in", "x", "dt", "o"))
        self.taps, self.conv_bias = w.vector(p + "conv"), w.vector(p + "conv.b")
        self.dt_bias, self.D = w.vector(p + "dt.b"), w.vector(p + "D")
        self.A = -torch.exp(w.vector(p + "A_log"))

    def register(self, state):
        state.register(self.key + ".conv", (self.taps_n - 1, self.inner))
        state.register(self.key + ".scan", (self.inner, self.n_states))

    def __call__(self, h, step):
        xz = linear(h, self.w_in)
        x = ops.conv_silu(xz[:, :self.inner], self.taps, self.conv_bias, step.state[self.key + ".conv"], step.spans)
        proj = linear_f32(x, self.w_x)
        dt = linear_f32(proj[:, :self.rank].to(x.dtype), self.w_dt)
        y = ops.selective_scan(x, xz[:, self.inner:], dt, self.dt_bias, self.A, proj[:, self.rank:], self.D,
                               step.state[self.key + ".scan"], step.spans)
        return linear(y, self.w_o)


class AttentionMixer:
    def __init__(self, w, p, m, config, key):
        self.m, self.eps, self.config = m, config.eps, config
        self.w_qkv, self.w_o = w.matrix(p + "q", p + "k", p + "v"), w.matrix(p + "o")
        self.q_norm, self.k_norm = w.vector(p + "q.norm"), w.vector(p + "k.norm")
        self.rot_dims = m["rot"]["dims"]
        self.key_freq = pair_frequencies(self.rot_dims, m["rot"]["base"], config.torch_device)
        self.value_freq = pair_frequencies(m["vdim"], m["rot"]["base"], config.torch_device)
        self.index = None  # of this layer's cache

    def register(self, state):
        pass

    def __call__(self, h, step):
        cache = step.caches[self.index]
        qkv = linear(h, self.w_qkv)
        positions = step.spans.positions
        q = cache.store_qkv(qkv, positions, self.q_norm, self.k_norm, self.eps, self.rot_dims, self.key_freq, self.value_freq,
                            append_tokens=step.append_tokens)
        o = cache.forward_rows(q, positions, self.value_freq, None if step.append_tokens is not None else step.spans.entry_of)
        return linear(o.view(o.shape[0], -1), self.w_o)


class LightningMixer:
    def __init__(self, w, p, m, config, key):
        self.heads, self.dim, self.vdim, self.key, self.eps = m["heads"], m["dim"], m["vdim"], key, config.eps
        self.w_qkvg, self.w_o, self.norm = w.matrix(p + "q", p + "k", p + "v", p + "g"), w.matrix(p + "o"), w.vector(p + "norm")
        self.decay = torch.tensor(m["decay"], dtype=torch.float32, device=config.torch_device)

    def register(self, state):
        state.register(self.key + ".decay", (self.heads, self.dim, self.vdim))

    def __call__(self, h, step):
        qkvg = linear(h, self.w_qkvg)
        o = ops.decay_attention(qkvg, self.decay, self.dim, self.vdim, step.state[self.key + ".decay"], step.spans)
        o = ops.norm_rows(o, self.norm, self.eps, h.dtype, gate=qkvg[:, qkvg.shape[1] - o.shape[1]:])
        return linear(o, self.w_o)


MIXERS = {"mamba1": MambaMixer, "attention": AttentionMixer, "lightning": LightningMixer}


class Layer:
    def __init__(self, w, i, spec, config):
        p = self.key = "l%d" % i
        self.eps = config.eps
        self.mu = w.vector(p + ".shift")
        self.mixer = MIXERS[spec["type"]](w, p + ".mix.", spec["mixer"], config, p)
        self.norm1, self.gate1, self.gate1_bias = w.vector(p + ".norm1"), w.matrix(p + ".rg1"), w.vector(p + ".rg1.b")
        self.has_ff = spec.get("mlp") is not None
        if self.has_ff:
            self.ff = spec["mlp"]["ff"]
            self.w_up_gate, self.w_down = w.matrix(p + ".mlp.up", p + ".rg2"), w.matrix(p + ".mlp.down")
            self.norm2, self.gate2_bias = w.vector(p + ".norm2"), w.vector(p + ".rg2.b")

    def register(self, state, config):
        state.register(self.key + ".shift", (config.width,))
        self.mixer.register(state)

    def __call__(self, x, plain, shifted, step, following):
        """x: fp32 stream, updated in place.  plain / shifted: x and its token shift in the model's dtype, when the
        layer before has left them.  Returns the same for `following`, the next layer."""
        if shifted is None:
            plain, shifted = ops.token_shift(x, self.mu, step.state[self.key + ".shift"], step.spans, step.dtype)
        r = self.mixer(shifted, step)
        gate = linear(plain, self.gate1)
        nxt = {}
        if step.spans.single and following is not None:  # one token per sequence: the sum also shifts for the next layer
            nxt = {"next_mu": following.mu, "next_state": step.state[following.key + ".shift"], "spans": step.spans}
        if not self.has_ff:
            return ops.gated_norm_add(x, r, gate, self.gate1_bias, self.norm1, self.eps, want_plain=bool(nxt), **nxt)
        plain, _ = ops.gated_norm_add(x, r, gate, self.gate1_bias, self.norm1, self.eps)
        up_gate = linear(plain, self.w_up_gate)
        r = linear(ops.gelu_tanh(up_gate[:, :self.ff]), self.w_down)
        return ops.gated_norm_add(x, r, up_gate[:, self.ff:], self.gate2_bias, self.norm2, self.eps, want_plain=bool(nxt), **nxt)


class Step:
    """What the layers of one step share."""

    def __init__(self, spans, caches, state, append_tokens, dtype):
        self.spans, self.caches, self.state, self.append_tokens, self.dtype = spans, caches, state, append_tokens, dtype


def random_weights(config, seed, device="cpu"):
    """Random tensors of the right names and shapes: matrices N(0, 1 / fan-in), Mamba's A and step sizes in their usual
    ranges, everything else near its neutral value."""
    g = torch.Generator(device=device).manual_seed(seed)
    W, out = config.width, {}

    def randn(*shape):
        return torch.randn(shape, generator=g, device=device)

    def matrix(name, rows, cols):
        out[name] = (randn(rows, cols) * cols ** -0.5).to(torch.bfloat16)

    def near(name, value, spread, *shape):
        out[name] = (value + spread * randn(*shape)).to(torch.bfloat16)

    out["embed"] = randn(config.vocab, W).to(torch.bfloat16)
    for i, spec in enumerate(config.layers):
        p, m = "l%d." % i, spec["mixer"]
        near(p + "norm1", 1.0, 0.1, W)
        near(p + "shift", 0.3, 0.2, W)
        matrix(p + "rg1", W, W)
        near(p + "rg1.b", 0.0, 0.5, W)
        x = p + "mix."
        if spec["type"] == "mamba1":
            C, N, R = m["inner"], m["state"], m["dt_rank"]
            matrix(x + "in", 2 * C, W)
            near(x + "conv", 0.0, 0.5, C, m["conv"])
            near(x + "conv.b", 0.0, 0.1, C)
            matrix(x + "x", R + 2 * N, C)
            matrix(x + "dt", C, R)
            near(x + "dt.b", -3.0, 1.0, C)
            out[x + "A_log"] = torch.log(torch.arange(1, N + 1, device=device).float()).repeat(C, 1).to(torch.bfloat16)
            near(x + "D", 1.0, 0.1, C)
            matrix(x + "o", W, C)
        elif spec["type"] == "attention":
            matrix(x + "q", m["heads"] * m["dim"], W)
            matrix(x + "k", m["kv_heads"] * m["dim"], W)
            matrix(x + "v", m["kv_heads"] * m["vdim"], W)
            near(x + "q.norm", 1.0, 0.1, m["dim"])
            near(x + "k.norm", 1.0, 0.1, m["dim"])
            matrix(x + "o", W, m["heads"] * m["vdim"])
        else:
            H = m["heads"]
            matrix(x + "q", H * m["dim"], W)
            matrix(x + "k", H * m["dim"], W)
            matrix(x + "v", H * m["vdim"], W)
            matrix(x + "g", H * m["vdim"], W)
            matrix(x + "o", W, H * m["vdim"])
            near(x + "norm", 1.0, 0.1, H * m["vdim"])
        if spec.get("mlp") is not None:
            near(p + "norm2", 1.0, 0.1, W)
            matrix(p + "rg2", W, W)
            near(p + "rg2.b", 0.0, 0.5, W)
            matrix(p + "mlp.up", spec["mlp"]["ff"], W)
            matrix(p + "mlp.down", W, spec["mlp"]["ff"])
    near("final.norm", 1.0, 0.1, W)
    matrix("head", config.vocab, W)
    return out


class GagoraxForCausalLM:
    def __init__(self, config: GagoraxConfig, tensors=None, seed=None):
        """`tensors`: the named weights (weights.read_model_weights); or a seed for random ones."""
        if tensors is None:
            tensors = random_weights(config, 0 if seed is None else seed)
        self.config = config
        self.device = torch.device(config.torch_device)
        # sums of products stay in fp32: no TF32, no 16-bit reductions between the parts of a split GEMM
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        w = Weights(tensors, config)
        self.embed = w.matrix("embed")
        self.layers = [Layer(w, i, spec, config) for i, spec in enumerate(config.layers)]
        self.final_norm, self.head = w.vector("final.norm"), w.matrix("head")
        self.attention_layers = [l.mixer for l in self.layers if isinstance(l.mixer, AttentionMixer)]
        for i, mixer in enumerate(self.attention_layers):
            mixer.index = i

    # ---- caches ----------------------------------------------------------------------------------------------------
    def create_kv_caches(self, max_tokens=None):
        """One Attention per attention layer, then the RecurrentState.  Pools hold `max_tokens` tokens each, or share the
        memory the configuration allows."""
        cfg = self.config
        state = RecurrentState(self.device, slots=cfg.state_slots)
        for layer in self.layers:
            layer.register(state, cfg)
        item = 2 if cfg.torch_dtype == torch.bfloat16 else 4
        per16 = 16 // item

        def chunk_bytes(m):
            pad = sum(-(-d // per16) * per16 for d in (m["dim"], m["vdim"]))
            return m["kv_heads"] * pad * cfg.chunk_size * item

        total = sum(chunk_bytes(a.m) for a in self.attention_layers)
        if max_tokens is not None:
            n_chunks = -(-max_tokens // cfg.chunk_size) + 64  # partly filled tails
        elif total:
            if cfg.kvcache_gb > 0:
                room = cfg.kvcache_gb * 2 ** 30
            else:
                room = 0.8 * torch.cuda.mem_get_info(self.device)[0]
            n_chunks = int(room // total)
        caches, made = [], {}
        for a in self.attention_layers:
            m = a.m
            key = (m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"])
            if key in made:  # same geometry: the layers share their work lists
                caches.append(chunk_attn.Attention(made[key]))
                continue
            made[key] = chunk_attn.Attention.shaped(
                n_heads=m["heads"], n_kv_heads=m["kv_heads"], d_key=m["dim"], d_value=m["vdim"], scale=m["scale"], sink=True,
                chunk_size=cfg.chunk_size, memory_mb=int(math.ceil(n_chunks * chunk_bytes(m) / 2 ** 20)), share_prefix=True,
                dtype=cfg.torch_dtype, device=self.device)
            caches.append(made[key])
        return caches + [state]

    # ---- one step --------------------------------------------------------------------------------------------------
    @torch.inference_mode()
    def step(self, rows, tokens, caches, tap=None):
        """Runs the next tokens of some sequences: entry i continues the sequence at row rows[i] of the caches with
        tokens[i], or starts a new one (None).  Returns (fp32 stream after the last layer, the spans, the rows): a new
        sequence's row is the one it was inserted at, as `Attention.add_seq` returns it.  tap(i, x): called after layer
        i with the stream."""
        state, attention = caches[-1], caches[:-1]
        decode = len(rows) == len(state) and all(r == i for i, r in enumerate(rows)) and all(len(t) == 1 for t in tokens)
        slots = [None if r is None else state.rows[r] for r in rows]
        out_rows = list(rows)
        if not decode:
            asked = [-1 if r is None else r for r in rows]
            got = None
            for cache in attention:
                r = cache.extend(asked, tokens)
                if got is not None and r != got:
                    raise RuntimeError("the layers' caches disagree about the rows")
                got = r
            for i, r in enumerate(rows):
                if r is None:
                    out_rows[i] = len(state) if got is None else got[i]
                    slots[i] = state.insert(out_rows[i])
        starts = [state.length[s] for s in slots]
        spans = SpanBatch(tokens, starts, slots, self.device)
        for s, t in zip(slots, tokens):
            state.length[s] += len(t)
        step = Step(spans, attention, state, [t[0] for t in tokens] if decode else None, self.config.torch_dtype)
        x = ops.embed_rows(self.embed, spans)
        plain = shifted = None
        for i, layer in enumerate(self.layers):
            plain, shifted = layer(x, plain, shifted, step, self.layers[i + 1] if i + 1 < len(self.layers) else None)
            if tap is not None:
                tap(i, x)
        return x, spans, out_rows

    @torch.inference_mode()
    def head_logits(self, x, rows):
        """fp32 logits of the given rows (int32 tensor) of a step's stream."""
        h = ops.norm_rows(x, self.final_norm, self.config.eps, self.config.torch_dtype, rows=rows)
        return linear_f32(h, self.head) * self.config.logit_scale

    # ---- the protocol of ModelHost -----------------------------------------------------------------------------------
    def _prefill(self, seqs, caches):
        """Runs whole prompts in portions of at most config.prefill_portion tokens; returns their last logits."""
        done, row_of = [0] * len(seqs), [None] * len(seqs)
        logits = [None] * len(seqs)
        while any(l is None for l in logits):
            budget, picked = self.config.prefill_portion, []
            for i, seq in enumerate(seqs):
                n = min(budget, len(seq) - done[i])
                if n > 0:
                    picked.append((i, n))
                    budget -= n
                if budget == 0:
                    break
            x, spans, rows = self.step([row_of[i] for i, _ in picked], [seqs[i].tokens[done[i]:done[i] + n] for i, n in picked], caches)
            for (i, n), r in zip(picked, rows):
                if row_of[i] is None:  # inserted: the rows at and after it have moved up
                    row_of = [None if q is None else q + (q >= r) for q in row_of]
                    row_of[i] = seqs[i].index = r
                done[i] += n
            ends = [k for k, (i, _) in enumerate(picked) if done[i] == len(seqs[i])]
            if ends:
                for k, row in zip(ends, self.head_logits(x, spans.last[ends])):
                    logits[picked[k][0]] = row
        return torch.stack(logits)

    @torch.inference_mode()
    def logits(self, seqs, kv_caches, prefill):
        """[n_seqs, vocab] scores of each sequence's next token."""
        if prefill:
            return self._prefill(seqs, kv_caches)
        x, spans, _ = self.step(list(range(len(seqs))), [[seq[-1]] for seq in seqs], kv_caches)
        return self.head_logits(x, spans.last)

    def __call__(self, seqs, kv_caches, prefill):
        return torch.argmax(self.logits(seqs, kv_caches, prefill), dim=-1).tolist()
