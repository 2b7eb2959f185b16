"""Decoders that run STEPS: what the models with an fp32 residual stream share.

A step brings the next tokens of any number of sequences (a whole prompt, a portion of one, a decoded token), laid end
to end; everything older comes from the caches.  Prefill, decode and continued portions are the same code; a step of one
token for every row takes the decode kernels, which walk shared prefixes once.  Call protocol as the Llama decoder's:
`model(seqs, kv_caches, prefill)` returns the next token of each sequence, `model.create_kv_caches()` makes the caches,
so `ModelHost` serves every such model unchanged.

The caches of a model are a list: any number of `chunk_attn.Attention`, whose rows move together, then one
`RecurrentState`, which also knows how many tokens each row has run.
"""
import torch
from torch.nn.functional import linear

from chunk_attn import SpanBatch


def linear_f32(x, w):
    """x W^T with the fp32 accumulator as the result."""
    if x.dtype == torch.float32:
        return linear(x, w)
    return torch.mm(x, w.t(), out_dtype=torch.float32)


def pair_frequencies(dims, base, device):
    """Radians per position of the dims / 2 rotation pairs, rounded once to fp32."""
    f = float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    return f.to(torch.float32).to(device)


def split_frequencies(dims, base, device):
    """[2, dims / 2]: the frequencies rounded to fp32, and what rounding left out."""
    f = float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    hi = f.to(torch.float32)
    return torch.stack([hi, (f - hi.double()).to(torch.float32)]).to(device)


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


class Step:
    """What the layers of one step share."""

    def __init__(self, spans, caches, state, append_tokens, dtype):
        self.spans, self.caches, self.state, self.append_tokens, self.dtype = spans, caches, state, append_tokens, dtype


class SpanDecoder:
    """A model provides run(step, tap) -> the fp32 stream after the last layer, head_logits(x, rows) and
    create_kv_caches(); the configuration's engine side is config.torch_dtype, torch_device and prefill_portion."""

    def __init__(self, config):
        self.config = config
        self.device = torch.device(config.torch_device)
        # sums of products stay in fp32: no TF32, no 16-bit reductions between the parts of a split GEMM
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False

    def appends(self, attention):
        """Whether the caches have decode kernels that append; otherwise a decoded token is a portion of one token."""
        return True

    # ---- one step --------------------------------------------------------------------------------------------------
    @torch.inference_mode()
    def step(self, rows, tokens, caches, tap=None):
        """Runs the next tokens of some sequences: entry i continues the sequence at row rows[i] of the caches with
        tokens[i], or starts a new one (None).  Returns (fp32 stream after the last layer, the spans, the rows): a new
        sequence's row is the one it was inserted at, as `Attention.add_seq` returns it.  tap(i, x): called after layer
        i with the stream."""
        state, attention = caches[-1], caches[:-1]
        decode = self.appends(attention) and len(rows) == len(state) and all(r == i for i, r in enumerate(rows)) and all(len(t) == 1 for t in tokens)
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
        x = self.run(step, tap)
        return x, spans, out_rows

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
