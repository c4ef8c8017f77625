"""Two mixers side by side on the same input.

y = factor * (rms_norm(left(h)) * w_left + rms_norm(right(h)) * w_right), the norms over the model width.  The two
share one input product: the rows of both mixers' input projections are one weight.  Their output projections are
two products (each output is normed by itself); the two norms and the sum run inside the kernel that writes the
result into the residual (``forward_pair``), or in a kernel of their own (``forward``).
"""

from __future__ import annotations

import torch

from ..ops import kernels, linear
from .base import BuildContext, ParamSpec, Part, kv_need, state_needs
from .hyper import NormedPair
from .registry import register_part


class ParallelMixers(Part):
    """``left`` and ``right`` are mixers that can be guests of a block (``input_rows``, ``output_cols``, ``between``);
    a guest may have a bias behind its output projection (``output_bias``, float32 [width])."""

    def __init__(self, ctx: BuildContext, *, hidden_size: int, left, right, eps: float, factor: float = 0.5,
                 left_name: str = "left", right_name: str = "right", norm_name: str = "out") -> None:
        self.hidden_size, self.eps, self.factor = hidden_size, float(eps), float(factor)
        self.left = ctx.build("mixer", left.with_params(hosted=True), ctx.child(left_name))
        self.right = ctx.build("mixer", right.with_params(hosted=True), ctx.child(right_name))
        self.norm_names = [f"{ctx.prefix}.{name}.{norm_name}" for name in (left_name, right_name)]
        for guest in (self.left, self.right):
            if not hasattr(guest, "between"):
                raise ValueError("mixers side by side share a product: both must be able to be a block's guests")
        self.in_weight = self.left_o_weight = self.right_o_weight = None
        self.left_norm_weight = self.right_norm_weight = None

    def children(self):
        return [self.left, self.right]

    def param_specs(self):
        (left_o, left_cols), (right_o, right_cols) = self.left.output_cols(), self.right.output_cols()
        return [ParamSpec.packed("in_weight", self.left.input_rows() + self.right.input_rows(), self.hidden_size),
                ParamSpec.single("left_o_weight", left_o, (self.hidden_size, left_cols)),
                ParamSpec.single("right_o_weight", right_o, (self.hidden_size, right_cols)),
                ParamSpec.single("left_norm_weight", self.norm_names[0], (self.hidden_size,), role="vector", init="around_one"),
                ParamSpec.single("right_norm_weight", self.norm_names[1], (self.hidden_size,), role="vector", init="around_one")]

    def finalize(self) -> None:
        self.left_norm_weight = self.left_norm_weight.to(torch.float32).contiguous()
        self.right_norm_weight = self.right_norm_weight.to(torch.float32).contiguous()

    def streamed_weights(self):
        return [self.in_weight, self.left_o_weight, self.right_o_weight]

    def cache_need(self):
        needs = [guest.cache_need() for guest in (self.left, self.right)]
        needs = tuple(n for need in needs for n in (need if isinstance(need, tuple) else (need,)) if n is not None)
        kv_need(needs), state_needs(needs)           # one cache at most, states with names of their own
        return needs

    def takes_tensor_memory_tiles(self, page_size: int) -> bool:
        asked = [getattr(guest, "takes_tensor_memory_tiles", None) for guest in (self.left, self.right)]
        return all(ask is not None and ask(page_size) for ask in asked)

    def scratch_floats(self, rows: int, chunks: int) -> int:
        asked = [getattr(guest, "scratch_floats", None) for guest in (self.left, self.right)]
        return max((ask(rows, chunks) for ask in asked if ask is not None), default=0)

    # ---------------------------------------------------------------- running
    def forward_pair(self, x, ctx, run: int) -> NormedPair:
        projected = linear(x, self.in_weight)
        outputs, at = [], 0
        for guest, o_weight in ((self.left, self.left_o_weight), (self.right, self.right_o_weight)):
            inner = torch.empty((x.shape[0], o_weight.shape[1]), dtype=x.dtype, device=x.device)
            guest.between(projected, at, ctx, inner, run)
            outputs.append(linear(inner, o_weight, out_dtype=torch.float32))
            at += sum(rows for _, rows in guest.input_rows())
        return NormedPair(outputs[0], outputs[1], left_weight=self.left_norm_weight,
                          right_weight=self.right_norm_weight, left_bias=getattr(self.left, "output_bias", None),
                          right_bias=getattr(self.right, "output_bias", None), eps=self.eps, factor=self.factor)

    def forward(self, x, ctx, run: int):
        return self.forward_pair(x, ctx, run).materialise()


register_part("mixer", "parallel_mixers", ParallelMixers)
