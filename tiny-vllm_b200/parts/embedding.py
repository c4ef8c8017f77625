"""Token embedding and the language-model head.

h = E[ids] (tinyvllm/models/qwen3.py:427-432, :480); logits = h . W^T with W the
embedding itself when tied (:514-525, :703-717).  Logits leave in float32.
"""

from __future__ import annotations

import torch

from ..ops import kernels, linear
from .base import EMBEDDING, BuildContext, ParamSpec, Part, StateNeed
from .registry import register_part


class TokenEmbedding(Part):
    """h = E[ids]; with ``norm`` (a norm part that offers ``start``) the rows are normed at once and leave
    in float32, as the first tensor of a float32 residual stream.  With ``stream_scale`` they are multiplied by it in
    float32 and start the stream as they are; the rows rounded to the storage type ride on it as ``rounded``."""

    def __init__(self, ctx: BuildContext, *, vocab_size: int, width: int, name: str, norm=None,
                 stream_scale: float | None = None) -> None:
        if norm is not None and stream_scale is not None:
            raise ValueError("an embedding is normed or scaled")
        self.vocab_size, self.width, self.name = vocab_size, width, name
        self.stream_scale = None if stream_scale is None else float(stream_scale)
        self.weight = None
        self.norm = ctx.build("norm", norm, ctx) if norm is not None else None
        if self.norm is not None and not hasattr(self.norm, "start"):
            raise ValueError("an embedding's norm must offer start(x)")

    def param_specs(self):
        return [ParamSpec.single("weight", self.name, (self.vocab_size, self.width), role="table")]

    def children(self):
        return [self.norm] if self.norm is not None else []

    def forward(self, token_ids):
        if self.stream_scale is not None:
            stream, rounded = kernels.embed_scaled(self.weight, token_ids, self.stream_scale)
            stream.rounded = rounded
            return stream
        rows = kernels.embed_rows(self.weight, token_ids)
        return rows if self.norm is None else self.norm.start(rows)


class PairEmbedding(Part):
    """h = E[token] + P[row] in float32, as the first tensor of a float32 stream; row = (previous * mul_prev + token *
    mul_cur) mod buckets is a hash of the pair (previous token, token), and a request's first token has the last
    row, number ``buckets``.  ``pairs``: {"buckets", "mul_prev", "mul_cur", "name"} or None for the plain rows.

    The token before is part of a request's state: one int32 a slot, left by every step as the last token of the
    entry."""

    def __init__(self, ctx: BuildContext, *, vocab_size: int, width: int, name: str, pairs: dict | None = None) -> None:
        self.vocab_size, self.width, self.name = vocab_size, width, name
        self.pairs = None if pairs is None else dict(pairs)
        self.weight = self.pair_weight = None

    def param_specs(self):
        specs = [ParamSpec.single("weight", self.name, (self.vocab_size, self.width), role="table")]
        if self.pairs is not None:
            specs.append(ParamSpec.single("pair_weight", self.pairs["name"], (self.pairs["buckets"] + 1, self.width),
                                          role="table"))
        return specs

    def state_need(self):
        return None if self.pairs is None else StateNeed((1,), torch.int32)

    def forward_step(self, ctx):
        hashed = None
        if self.pairs is not None:
            hashed = dict(table=self.pair_weight, mul_prev=self.pairs["mul_prev"], mul_cur=self.pairs["mul_cur"],
                          state=ctx.storage.state_of(EMBEDDING))
        return kernels.embed_pairs(self.weight, ctx.token_ids, positions=ctx.positions, token_row=ctx.token_row,
                                   row_starts=ctx.row_starts, state_slots=ctx.state_slots, pairs=hashed)


class LMHead(Part):
    def __init__(self, ctx: BuildContext, *, vocab_size: int, width: int, name: str,
                 tied_to: str | None, scale: float = 1.0) -> None:
        self.vocab_size, self.width, self.name, self.tied_to = vocab_size, width, name, tied_to
        self.scale = float(scale)          # the float32 logits are multiplied by it
        self.weight = None

    def param_specs(self):
        if self.tied_to is not None:
            return []
        return [ParamSpec.single("weight", self.name, (self.vocab_size, self.width))]

    def streamed_weights(self):
        return [self.weight]

    def forward(self, hidden_rows):
        logits = linear(hidden_rows, self.weight, out_dtype=torch.float32)
        return logits if self.scale == 1.0 else kernels.scale_float32(logits, self.scale)


register_part("embedding", "token_embedding", TokenEmbedding)
register_part("embedding", "pair_embedding", PairEmbedding)
register_part("head", "lm_head", LMHead)
