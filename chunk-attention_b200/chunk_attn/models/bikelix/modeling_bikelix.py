"""Bikelix: a decoder of windowed latent-attention layers with shared latent caches over one fp32 residual stream.

A layer is x = norm(alpha x + mixer(x)) and, when it has a feed-forward, x = norm(alpha x + ff(x)).  Tensors are named
`embed`, `l<i>.norm1`, `l<i>.mix.*`, `l<i>.norm2`, `l<i>.mlp.*`, `final.norm`; the head is the embedding table.

What attention keeps of a token is one row for all heads: a normalised latent c and a rotated key part k_r.  With
k_h = (U_h c, k_r) and v_h = W_h c the scores are q_h . k_h = (U_h^T q_h) . c + q_r . k_r, so there are two ways to run a
layer on the cached rows:
  absorbed   the queries go into the latent space (U_h^T q_h), attention works on the rows themselves, and W_h is applied
             to its result.  Every row is read once for all heads: decode, and short portions behind a long context
  expanded   keys and values of every head are made from the rows of the step's windows by one GEMM, then attended to
             with their own, smaller sizes: prompts
A layer may read the cache of an earlier one (`kv_from`) with queries, projections, scale and window of its own: it holds
a reader of that layer's `chunk_attn.Attention`.
"""
import math

import torch
from torch.nn.functional import linear

import chunk_attn
from chunk_attn import ops

from ..recurrent_state import RecurrentState
from ..span_decoder import SpanDecoder, Weights, linear_f32, split_frequencies
from .configuration_bikelix import BikelixConfig

GATE_SLOPE = 1.702
EXPAND_MIN_TOKENS = 32   # of a step
ABSORBED_COST = 2        # of a product in the latent space, in units of one between expanded heads


class LatentAttentionMixer:
    def __init__(self, w, p, m, config, layer):
        self.m, self.eps, self.layer = m, config.eps, layer
        self.heads, self.dim, self.rot, self.vdim = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
        self.owner = m.get("kv_from")  # None: this layer stores rows of its own
        if self.owner is None:
            self.w_in, self.kv_norm = w.matrix(p + "dq", p + "dkv"), w.vector(p + "dkv.norm")
        else:
            self.w_in = w.matrix(p + "dq")
        self.q_norm, self.w_uq, self.w_o = w.vector(p + "dq.norm"), w.matrix(p + "uq"), w.matrix(p + "o")
        uk, uv = w.matrix(p + "uk"), w.matrix(p + "uv")
        self.w_ukv = torch.cat([uk, uv])  # [heads * (dim + vdim), latent]: the expansion
        self.w_uk = self.w_ukv[:uk.shape[0]].view(self.heads, self.dim, m["kv_rank"])
        self.w_uv = self.w_ukv[uk.shape[0]:].view(self.heads, self.vdim, m["kv_rank"])
        self.sink = w.vector(p + "sink")
        self.freq = split_frequencies(self.rot, m["rot"]["base"], config.torch_device)
        self.cache = None

    def geometry(self):
        m = self.m
        return (m["heads"], m["kv_rank"], m["rot_dim"], m["scale"], m["mask"]["size"])

    def queries(self, h, step, cache):
        """[tokens, heads, dim + rot_dim], the last part not rotated yet; a layer of its own rows stores them on the way."""
        x = linear(h, self.w_in)
        if self.owner is None:
            c = cache.store_latent(x, step.spans.positions, self.q_norm, self.kv_norm, self.eps, self.freq, append_tokens=step.append_tokens)
        else:
            c = ops.norm_rows(x, self.q_norm, self.eps, x.dtype)
        return linear(c, self.w_uq).view(-1, self.heads, self.dim + self.rot)

    def absorbed(self, q, step, cache):
        T = q.shape[0]
        q_lat = torch.empty(T, self.heads, self.m["kv_rank"], dtype=q.dtype, device=q.device)
        torch.bmm(q[..., :self.dim].transpose(0, 1), self.w_uk, out=q_lat.transpose(0, 1))
        c = cache.forward_latent(q_lat, q, step.spans.positions, self.freq, self.sink,
                                 None if step.append_tokens is not None else step.spans.entry_of)
        o = torch.empty(T, self.heads, self.vdim, dtype=q.dtype, device=q.device)
        torch.bmm(c.transpose(0, 1), self.w_uv.transpose(1, 2), out=o.transpose(0, 1))
        return o

    def expanded(self, q, step, cache):
        lat, rot = cache.gather_latents()
        return cache.forward_expanded(q, linear(lat, self.w_ukv), rot, step.spans.positions, self.freq, self.sink, self.vdim)

    def expands(self, tokens, step, cache):
        """Whether making keys and values of the step's windows is less work than bringing its queries into the latent
        space and attending there, on whose longer rows the tensor cores also run slower."""
        if step.append_tokens is not None or tokens < EXPAND_MIN_TOKENS or not cache.latent_expands(self.dim, self.vdim):
            return False
        rows, pairs = cache.window_load()
        per_row = self.m["kv_rank"] * (self.dim + self.vdim)
        there = ABSORBED_COST * pairs * (2 * self.m["kv_rank"] + self.rot)
        return rows * per_row + pairs * (self.dim + self.rot + self.vdim) < tokens * per_row + there

    def __call__(self, h, step):
        cache = step.state.views[self.layer]
        q = self.queries(h, step, cache)
        attend = self.expanded if self.expands(q.shape[0], step, cache) else self.absorbed
        o = attend(q, step, cache)
        return linear(o.view(o.shape[0], -1), self.w_o)


class ClampedGLU:
    """Gated linear unit of clamped halves with biases; the last bias is left to the norm that follows."""

    def __init__(self, w, p, spec):
        self.limit = spec["limit"]
        self.w_gate_up, self.w_down = w.matrix(p + "gate", p + "up"), w.matrix(p + "down")
        self.gate_up_bias = torch.cat([w.vector(p + "gate.b"), w.vector(p + "up.b")])
        self.bias = w.vector(p + "down.b")

    def __call__(self, h):
        return linear(ops.clamped_glu(linear(h, self.w_gate_up), self.gate_up_bias, self.limit, GATE_SLOPE), self.w_down)


MIXERS = {"latent_attention": LatentAttentionMixer}
FEED_FORWARDS = {"dense": ClampedGLU}


class Layer:
    def __init__(self, w, i, spec, config):
        p = "l%d." % i
        self.alpha, self.eps = config.postln_alpha, config.eps
        self.mixer = MIXERS[spec["type"]](w, p + "mix.", spec["mixer"], config, i)
        self.norm1 = w.vector(p + "norm1") + 1.0  # weights are stored as distances from one
        self.ff = None
        if spec.get("mlp") is not None:
            self.ff = FEED_FORWARDS[spec["mlp"]["kind"]](w, p + "mlp.", spec["mlp"])
            self.norm2 = w.vector(p + "norm2") + 1.0

    def __call__(self, x, h, step):
        """x: fp32 stream, updated in place; h: x in the model's dtype.  Returns the new h."""
        h = ops.scaled_norm(x, self.mixer(h, step), self.alpha, self.norm1, self.eps)
        if self.ff is not None:
            h = ops.scaled_norm(x, self.ff(h), self.alpha, self.norm2, self.eps, bias=self.ff.bias)
        return h


def random_weights(config, seed, device="cpu"):
    """Random tensors of the right names and shapes: matrices N(0, 1 / fan-in), everything else near its neutral value."""
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
        x, H = p + "mix.", m["heads"]
        near(p + "norm1", 0.0, 0.1, W)
        matrix(x + "dq", m["q_rank"], W)
        near(x + "dq.norm", 1.0, 0.1, m["q_rank"])
        matrix(x + "uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"])
        if m.get("kv_from") is None:
            matrix(x + "dkv", m["kv_rank"] + m["rot_dim"], W)
            near(x + "dkv.norm", 1.0, 0.1, m["kv_rank"])
        matrix(x + "uk", H * m["dim"], m["kv_rank"])
        matrix(x + "uv", H * m["vdim"], m["kv_rank"])
        near(x + "sink", 0.0, 1.0, H)
        matrix(x + "o", W, H * m["vdim"])
        if spec.get("mlp") is not None:
            F = spec["mlp"]["ff"]
            near(p + "norm2", 0.0, 0.1, W)
            for name, rows, cols in (("gate", F, W), ("up", F, W), ("down", W, F)):
                matrix(p + "mlp." + name, rows, cols)
                near(p + "mlp." + name + ".b", 0.0, 0.2, rows)
    near("final.norm", 0.0, 0.1, W)
    return out


class BikelixForCausalLM(SpanDecoder):
    def __init__(self, config: BikelixConfig, tensors=None, seed=None):
        """`tensors`: the named weights (weights.read_model_weights); or a seed for random ones."""
        if tensors is None:
            tensors = random_weights(config, 0 if seed is None else seed)
        super().__init__(config)
        w = Weights(tensors, config)
        self.embed = w.matrix("embed")
        self.layers = [Layer(w, i, spec, config) for i, spec in enumerate(config.layers)]
        self.final_norm = w.vector("final.norm") + 1.0

    # ---- caches ----------------------------------------------------------------------------------------------------
    def create_kv_caches(self, max_tokens=None):
        """One Attention per layer that stores rows, then the RecurrentState (which only counts tokens here).  Pools hold
        `max_tokens` tokens each, or share the memory the configuration allows.  Layers that read another layer's cache
        have a reader of it, kept beside the caches in `state.views`."""
        cfg = self.config
        item = 2 if cfg.torch_dtype == torch.bfloat16 else 4
        line = 128 // item
        mixers = [l.mixer for l in self.layers]

        def chunk_bytes(m):
            return -(-(m["kv_rank"] + m["rot_dim"]) // line) * 128 * cfg.chunk_size

        total = sum(chunk_bytes(a.m) for a in mixers if a.owner is None)
        if max_tokens is not None:
            n_chunks = -(-max_tokens // cfg.chunk_size) + 64  # partly filled tails
        else:
            room = cfg.kvcache_gb * 2 ** 30 if cfg.kvcache_gb > 0 else 0.8 * torch.cuda.mem_get_info(self.device)[0]
            n_chunks = int(room // total)
        views, made, made_readers, owned = [], {}, {}, {}
        for i, a in enumerate(mixers):
            key = a.geometry()
            heads, latent, rotated, scale, window = key
            if a.owner is not None:
                reader = owned[a.owner].reader(n_heads=heads, scale=scale, window=window, sibling=made_readers.get(key))
                made_readers.setdefault(key, reader)
                views.append(reader)
                continue
            if key in made:  # same geometry: the layers share their work lists
                cache = chunk_attn.Attention(made[key])
            else:
                cache = made[key] = chunk_attn.Attention.latent(
                    n_heads=heads, latent=latent, rotated=rotated, scale=scale, window=window, chunk_size=cfg.chunk_size,
                    memory_mb=int(math.ceil(n_chunks * chunk_bytes(a.m) / 2 ** 20)), share_prefix=True, dtype=cfg.torch_dtype,
                    device=self.device)
            owned[i] = cache
            views.append(cache)
        state = RecurrentState(self.device, slots=cfg.state_slots)
        state.views = views
        return list(owned.values()) + [state]

    def appends(self, attention):
        return all(c.latent_decodes for c in attention)

    # ---- one step --------------------------------------------------------------------------------------------------
    def run(self, step, tap):
        if self.config.torch_dtype == torch.float32:
            x = h = ops.embed_rows(self.embed, step.spans, scale=self.config.embedding["scale"])
        else:
            x, h = ops.embed_rows(self.embed, step.spans, scale=self.config.embedding["scale"], want_plain=True)
        for i, layer in enumerate(self.layers):
            h = layer(x, h, step)
            if tap is not None:
                tap(i, x)
        return x

    @torch.inference_mode()
    def head_logits(self, x, rows):
        """fp32 logits of the given rows (int32 tensor) of a step's stream; the head is the embedding table."""
        h = ops.norm_rows(x, self.final_norm, self.config.eps, self.config.torch_dtype, rows=rows)
        return ops.softcap(linear_f32(h, self.embed), self.config.logit_softcap)
