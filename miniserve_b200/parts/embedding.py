"""Token embedding and the output head."""

from __future__ import annotations

import torch

from .. import ops
from .base import FixedState, Part, WeightDecl, param, register_part


@register_part("embedding", "token_embedding")
class TokenEmbedding(Part):
    """h = table[ids] (miniserve/model/qwen3.py:211), widened to the float32 residual stream.
    Parameters: ``vocab``, ``hidden``, ``name`` (the tensor's full name)."""
    shape_static = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.vocab = param(spec, "vocab", int)
        self.hidden = param(spec, "hidden", int)
        self.name = param(spec, "name", str)

    def weights(self):
        return {self.name: WeightDecl((self.vocab, self.hidden))}

    def bind(self, tensors):
        self.table = tensors[self.name].contiguous()

    def forward(self, ctx) -> torch.Tensor:
        residual = torch.empty((ctx.num_tokens, self.hidden), dtype=torch.float32, device=self.table.device)
        ops.embed_gather(residual, self.table, ctx.token_ids, stream=ctx.stream)
        return residual


@register_part("embedding", "summed_embedding")
class SummedEmbedding(Part):
    """h = scale * table[id] (+ bigram[row]) (+ sinusoid(position)), summed in float32 by one kernel.

    ``bigram`` (a mapping with ``buckets``, ``mul_prev``, ``mul_cur``, ``name``; or absent): a second table of buckets + 1 rows, read
    at row (previous token * mul_prev + token * mul_cur) mod buckets, and at its last row for a sequence's first token. The
    previous token is state of the request (one int32 in its slot), so that a portion or a decoded token continues from it.
    ``sinusoid`` (a base, or absent): entry 2i of the position's vector is sin(position * base^(-2i / hidden)), entry 2i + 1 the
    cosine (frequencies worked out in float64 and rounded once; the angle and its sine and cosine are float32).
    Parameters: ``vocab``, ``hidden``, ``name`` (the table's full name), ``bigram``, ``sinusoid``, ``scale`` (1)."""
    shape_static = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.vocab = param(spec, "vocab", int)
        self.hidden = param(spec, "hidden", int)
        self.name = param(spec, "name", str)
        self.scale = float(spec.params.get("scale", 1.0))
        b = spec.get("bigram")
        self.pair = (int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])) if b else None
        self.pair_name = str(b["name"]) if b else None
        if self.pair and (self.pair[0] < 1 or min(self.pair[1:]) < 0):
            raise ValueError(f"summed_embedding: a bigram table needs buckets and factors that are not negative, got {self.pair}")
        base = spec.get("sinusoid")
        self.inv_freq = None
        if base is not None:
            i = torch.arange(0, (self.hidden + 1) // 2, dtype=torch.float64)
            self.inv_freq = (float(base) ** (-2.0 * i / self.hidden)).to(torch.float32).to(env.device)

    def cache_need(self):
        return FixedState((1,), torch.int32) if self.pair else None

    def weights(self):
        w = {self.name: WeightDecl((self.vocab, self.hidden))}
        if self.pair:
            w[self.pair_name] = WeightDecl((self.pair[0] + 1, self.hidden))
        return w

    def bind(self, tensors):
        self.table = tensors[self.name].contiguous()
        self.pair_table = tensors[self.pair_name].contiguous() if self.pair else None

    def forward(self, ctx, cache=None) -> torch.Tensor:
        residual = torch.empty((ctx.num_tokens, self.hidden), dtype=torch.float32, device=self.table.device)
        ops.embed_sum(residual, self.table, ctx, self.inv_freq, self.pair_table, self.pair, cache.state if self.pair else None,
                      scale=self.scale)
        return residual


@register_part("head", "linear_head")
class LinearHead(Part):
    """logits = x @ W^T, no bias (miniserve/model/qwen3.py:186); with ``tied`` the matrix is the
    embedding table itself and no tensor of its own is read (miniserve/model/weights.py:116-119,
    135-136). Logits are returned in float32. Parameters: ``vocab``, ``hidden``, ``tied``,
    ``name``, ``tied_to``, optional ``scale`` (the float32 logits are multiplied by it)
    and ``softcap`` (then logits become softcap * tanh(logits / softcap))."""
    shape_static = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.vocab = param(spec, "vocab", int)
        self.hidden = param(spec, "hidden", int)
        self.tied = bool(spec.get("tied", False))
        self.name = param(spec, "name", str)
        self.tied_to = spec.get("tied_to")
        self.scale = float(spec.get("scale") or 1.0)
        self.softcap = float(spec.get("softcap") or 0.0)
        if self.softcap < 0:
            raise ValueError(f"a head's softcap={self.softcap} must not be negative")
        if self.tied and not self.tied_to:
            raise ValueError("a tied head needs 'tied_to', the name of the embedding tensor")

    def weights(self):
        return {} if self.tied else {self.name: WeightDecl((self.vocab, self.hidden))}

    def bind(self, tensors):
        if not self.tied:
            self.weight = tensors[self.name].contiguous()

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        logits = torch.empty((x.shape[0], self.vocab), dtype=torch.float32, device=x.device)
        if x.shape[0]:
            ops.linear(x, self.weight, out=logits, stream=ctx.stream)
            if self.scale != 1.0:
                ops.scale_(logits, self.scale, stream=ctx.stream)
            if self.softcap:
                ops.tanh_(logits, self.softcap, stream=ctx.stream)
        return logits
