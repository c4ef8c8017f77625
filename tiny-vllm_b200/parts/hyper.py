"""A residual of several streams, and the block over it (hyper-connections).

Instead of one residual x there are s copies x_1 .. x_s, all equal to the embedding at the start.  A sublayer reads
u = sum_s in[s] x_s; its output y is written back together with a mixing of the streams,
x_t <- sum_s mix[s, t] x_s + out[t] y, all streams at once from the old ones.  At the end x is the sum of the
streams.  Streams, mixing and norms are float32 whatever the storage type.

The write behind a sublayer and the norm in front of the next are one kernel: a block leaves its last write on
the stream tensor as ``stream.pending`` (:class:`HyperUpdate`), and whoever norms the streams next does it in the
same pass.  While all streams still equal the embedding the stream tensor is [tokens, width]; from the first
write on it is [tokens, streams, width].
"""

from __future__ import annotations

import torch

from ..ops import kernels
from .base import Block, BuildContext, ParamSpec, Part
from .registry import register_part


class NormedPair:
    """What two sublayers side by side left, not added up yet: factor * (norm(left) * left_weight + norm(right) *
    right_weight), norm dividing by the root mean square (``eps`` inside the root).  ``left`` and ``right`` are
    [tokens, width] of one dtype; the biases (float32 [width], or None) are added to them first."""

    __slots__ = ("left", "right", "left_weight", "right_weight", "left_bias", "right_bias", "eps", "factor")

    def __init__(self, left, right, *, left_weight, right_weight, left_bias=None, right_bias=None, eps, factor) -> None:
        self.left, self.right = left, right
        self.left_weight, self.right_weight = left_weight, right_weight
        self.left_bias, self.right_bias = left_bias, right_bias
        self.eps, self.factor = eps, factor

    def materialise(self):
        """The float32 sum itself."""
        return kernels.normed_pair_sum(self)


class HyperUpdate:
    """A write that is still to be done: ``y`` (a tensor or a :class:`NormedPair`) through ``connection``."""

    __slots__ = ("y", "connection")

    def __init__(self, y, connection) -> None:
        self.y, self.connection = y, connection


class HyperConnection(Part):
    """The stored numbers of one sublayer: ``in`` [streams], ``mix`` [streams, streams] (from, to), ``out`` [streams]."""

    def __init__(self, ctx: BuildContext, *, streams: int) -> None:
        self.streams = streams
        self.prefix = ctx.prefix
        self.w_in = self.w_mix = self.w_out = None

    def param_specs(self):
        return [ParamSpec.single("w_in", f"{self.prefix}.in", (self.streams,), role="vector", init="even"),
                ParamSpec.single("w_mix", f"{self.prefix}.mix", (self.streams, self.streams), role="vector", init="even"),
                ParamSpec.single("w_out", f"{self.prefix}.out", (self.streams,), role="vector", init="around_one")]

    def finalize(self) -> None:
        for attr in ("w_in", "w_mix", "w_out"):
            setattr(self, attr, getattr(self, attr).to(torch.float32).contiguous())


class HyperLayerNorm(Part):
    """Layer norm with weight and bias of what a sublayer reads from the streams, (u - mean) / sqrt(mean squared
    deviation + eps) * w + b, rounded once to the storage type; the write that is pending on the streams is done in
    the same pass.  The bias is the tensor of the weight's name with ".b" added."""

    def __init__(self, ctx: BuildContext, *, width: int, eps: float, name: str | None = None) -> None:
        self.width, self.eps = width, float(eps)
        self.name = name if name is not None else f"{ctx.prefix}.weight"
        self.out_dtype = ctx.dtype
        self.weight = self.bias = None

    def param_specs(self):
        return [ParamSpec.single("weight", self.name, (self.width,), role="vector", init="around_one"),
                ParamSpec.single("bias", f"{self.name}.b", (self.width,), role="vector")]

    def finalize(self) -> None:
        self.weight = self.weight.to(torch.float32).contiguous()
        self.bias = self.bias.to(torch.float32).contiguous()

    def read(self, stream, connection):
        """(norm of sum_s in[s] x_s, the streams after the pending write)."""
        pending = getattr(stream, "pending", None)
        return kernels.hyper_norm(stream, streams=connection.streams, w_in=connection.w_in, weight=self.weight,
                                  bias=self.bias, eps=self.eps, out_dtype=self.out_dtype,
                                  y=None if pending is None else pending.y,
                                  w_mix=None if pending is None else pending.connection.w_mix,
                                  w_out=None if pending is None else pending.connection.w_out)

    def add_rows(self, x, residual, rows):
        """The model's last norm: of the sum of the streams, on the rows named by ``rows`` only."""
        stream = x if residual is None else residual
        pending = getattr(stream, "pending", None)
        if pending is None or (residual is not None and x is not None):
            raise kernels.KernelError("this norm ends a model whose blocks leave a write pending on the streams")
        connection = pending.connection
        return kernels.hyper_norm(stream, streams=connection.streams, w_in=None, weight=self.weight, bias=self.bias,
                                  eps=self.eps, out_dtype=self.out_dtype, y=pending.y, w_mix=connection.w_mix,
                                  w_out=connection.w_out, rows=rows)[0]


class HyperResidualBlock(Block):
    """Pre-norm sublayers over a residual of ``streams`` streams; a layer may have no feed-forward.  A mixer may
    offer ``forward_pair(x, ctx, run)`` and return a :class:`NormedPair`, which the write adds up.  The block
    returns (None, stream) with the last write pending."""

    def __init__(self, ctx: BuildContext, *, mixer, feed_forward, norm, streams: int, mixer_norm_name: str,
                 feed_forward_norm_name: str, mixer_connection_name: str, feed_forward_connection_name: str,
                 mixer_name: str, feed_forward_name: str) -> None:
        def build_norm(name):
            return ctx.build("norm", norm.with_params(name=f"{ctx.prefix}.{name}"), ctx)

        self.mixer_norm = build_norm(mixer_norm_name)
        self.mixer_connection = HyperConnection(ctx.child(mixer_connection_name), streams=streams)
        self.mixer = ctx.build("mixer", mixer, ctx.child(mixer_name))
        self.feed_forward_norm = self.feed_forward_connection = self.feed_forward = None
        if feed_forward is not None:
            self.feed_forward_norm = build_norm(feed_forward_norm_name)
            self.feed_forward_connection = HyperConnection(ctx.child(feed_forward_connection_name), streams=streams)
            self.feed_forward = ctx.build("feed_forward", feed_forward, ctx.child(feed_forward_name))
        if not hasattr(self.mixer_norm, "read"):
            raise ValueError("a block over several streams needs norms that offer read(stream, connection)")

    def children(self):
        return [part for part in (self.mixer_norm, self.mixer_connection, self.mixer, self.feed_forward_norm,
                                  self.feed_forward_connection, self.feed_forward) if part is not None]

    def forward(self, hidden, residual, ctx, run: int):
        if residual is not None and hidden is not None:
            raise ValueError("a block over several streams follows blocks that leave nothing but the streams")
        stream = hidden if residual is None else residual
        x, stream = self.mixer_norm.read(stream, self.mixer_connection)
        pair = getattr(self.mixer, "forward_pair", None)
        stream.pending = HyperUpdate(pair(x, ctx, run) if pair is not None else self.mixer.forward(x, ctx, run),
                                     self.mixer_connection)
        if self.feed_forward is not None:
            x, stream = self.feed_forward_norm.read(stream, self.feed_forward_connection)
            stream.pending = HyperUpdate(self.feed_forward.forward(x, ctx), self.feed_forward_connection)
        return None, stream


register_part("norm", "layer_norm_hyper32", HyperLayerNorm)
register_part("block", "hyper_residual", HyperResidualBlock)
