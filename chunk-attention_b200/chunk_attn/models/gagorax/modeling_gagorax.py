"""Gagorax: a decoder of Mamba, rotary attention and linear-attention layers over one fp32 residual stream.

A layer is x += norm(gate * mixer(shift(x))) and, when it has a feed-forward, x += norm(gate * ff(x)): the sublayers
read the stream itself, the RMS norm is on their output.  Tensors are named `embed`, `l<i>.norm1`, `l<i>.shift`,
`l<i>.rg1`, `l<i>.mix.*`, `l<i>.mlp.*`, ..., `final.norm`, `head`.

The model runs steps (`SpanDecoder`); what a step reads of earlier tokens comes from the caches: one
`chunk_attn.Attention` per attention layer, one `RecurrentState` for the rest (shifted rows, convolution windows, scan
and linear-attention states).

Per sublayer: projections are library GEMMs with their weights concatenated where they read the same rows; everything
between them is a kernel of `chunk_attn.ops` or of the cache, with fp32 arithmetic on the residual, norms, angles,
scores, gates, step sizes and states.
"""
import math

import torch
from torch.nn.functional import linear

import chunk_attn
from chunk_attn import ops

from ..recurrent_state import RecurrentState
from ..span_decoder import SpanDecoder, Weights, linear_f32, pair_frequencies
from .configuration_gagorax import GagoraxConfig


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


class GagoraxForCausalLM(SpanDecoder):
    def __init__(self, config: GagoraxConfig, tensors=None, seed=None):
        """`tensors`: the named weights (weights.read_model_weights); or a seed for random ones."""
        if tensors is None:
            tensors = random_weights(config, 0 if seed is None else seed)
        super().__init__(config)
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
    def run(self, step, tap):
        x = ops.embed_rows(self.embed, step.spans)
        plain = shifted = None
        for i, layer in enumerate(self.layers):
            plain, shifted = layer(x, plain, shifted, step, self.layers[i + 1] if i + 1 < len(self.layers) else None)
            if tap is not None:
                tap(i, x)
        return x

    @torch.inference_mode()
    def head_logits(self, x, rows):
        """fp32 logits of the given rows (int32 tensor) of a step's stream."""
        h = ops.norm_rows(x, self.final_norm, self.config.eps, self.config.torch_dtype, rows=rows)
        return linear_f32(h, self.head) * self.config.logit_scale
