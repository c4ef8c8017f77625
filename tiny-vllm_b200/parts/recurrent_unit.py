"""A linear recurrent unit with gates (Griffin's recurrent block): one number of state a channel.

Two branches of ``channels``: y = W_y h + b_y, and u, a causal convolution over the last ``taps`` tokens of W_x h + b_x,
a channel by itself, with a bias and no activation (the inputs before a request's start are zeros, not biases).  u is
cut into ``blocks`` equal parts, and in each r = sigmoid(A_r u + b_r), i = sigmoid(A_i u + b_i) with square matrices of
the part's size; log a = -``decay_power`` * r * softplus(lam).  Per request a float32 state S [channels] runs along the
tokens: S <- a S + sqrt(1 - a^2) i u; the output is W_o (S * act(y)).

The mixer's memory is the state and the convolution's last inputs, a slot a request each in the cache storage's state
arenas.  Gates, decays, state and sums are float32 whatever the storage type.
"""

from __future__ import annotations

import torch

from ..ops import kernels, linear
from .base import BuildContext, ParamSpec, Part, StateNeed
from .registry import register_part


class LinearRecurrentUnit(Part):
    def __init__(self, ctx: BuildContext, *, hidden_size: int, channels: int, blocks: int, taps: int,
                 decay_power: float = 8.0, activation: str | None = "gelu_tanh", float32_output: bool = False,
                 names: dict | None = None) -> None:
        if blocks <= 0 or channels % blocks:
            raise ValueError("the unit's channels form equal blocks")
        if not 0 < taps <= kernels.CONV_TAPS[-1]:
            raise ValueError(f"the convolution takes up to {kernels.CONV_TAPS[-1]} taps, not {taps}")
        if activation not in kernels.UNIT_ACTS:
            raise ValueError(f"activation is None, 'silu' or 'gelu_tanh', not {activation!r}")
        self.hidden_size, self.channels, self.blocks, self.taps = hidden_size, channels, blocks, taps
        self.size = channels // blocks
        self.decay_power, self.activation = float(decay_power), activation
        self.out_dtype = torch.float32 if float32_output else None
        n = {"y": "y", "y_bias": "y.b", "x": "x", "x_bias": "x.b", "conv": "conv", "conv_bias": "conv.b", "r": "ra",
             "r_bias": "ra.b", "i": "ri", "i_bias": "ri.b", "lam": "lam", "o": "o", **(names or {})}
        self.names = {key: f"{ctx.prefix}.{value}" for key, value in n.items()}
        self.unit_state, self.conv_state = f"{ctx.prefix}.unit", f"{ctx.prefix}.conv"
        self.conv_taps = next(k for k in kernels.CONV_TAPS if k >= taps)
        self.in_weight = self.o_weight = self.y_bias = self.x_bias = self.conv_weight = self.conv_bias = None
        self.r_weight = self.r_bias = self.i_weight = self.i_bias = self.lam = None
        self.gate_weight = self.conv_by_tap = self.decay = None

    # ------------------------------------------------------------ declaration
    def param_specs(self):
        n, c, blocks, size = self.names, self.channels, self.blocks, self.size
        specs = [ParamSpec.packed("in_weight", [(n["x"], c), (n["y"], c)], self.hidden_size),
                 ParamSpec.single("o_weight", n["o"], (self.hidden_size, c)),
                 ParamSpec.single("conv_weight", n["conv"], (c, self.taps), role="vector", init="unit_interval"),
                 ParamSpec.single("lam", n["lam"], (c,), role="vector")]
        specs += [ParamSpec.single(attr, n[attr], (c,), role="vector") for attr in ("y_bias", "x_bias", "conv_bias")]
        for gate in ("r", "i"):
            specs += [ParamSpec.single(f"{gate}_weight", n[gate], (blocks, size, size)),
                      ParamSpec.single(f"{gate}_bias", n[f"{gate}_bias"], (blocks, size), role="vector")]
        return specs

    def finalize(self) -> None:
        """What the kernels read: taps by age with the missing older ones as zeros, the decay -power * softplus(lam),
        biases, all in float32, and both gates' matrices of a block as the rows of one."""
        if self.conv_by_tap is not None or self.conv_weight is None:
            return
        f32 = torch.float32
        self.conv_by_tap = torch.zeros((self.conv_taps, self.channels), dtype=f32, device=self.conv_weight.device)
        self.conv_by_tap[self.conv_taps - self.taps:] = self.conv_weight.to(f32).t()
        lam = self.lam.double()
        self.decay = (-self.decay_power * (lam.clamp(min=0) + torch.log1p(torch.exp(-lam.abs())))).to(f32).contiguous()
        for attr in ("y_bias", "x_bias", "conv_bias", "r_bias", "i_bias"):
            setattr(self, attr, getattr(self, attr).to(f32).flatten().contiguous())
        self.gate_weight = torch.cat([self.r_weight, self.i_weight], dim=1).contiguous()
        self.conv_weight = self.r_weight = self.i_weight = self.lam = None

    def streamed_weights(self):
        return [self.in_weight, self.o_weight]

    def cache_need(self):
        return (StateNeed((self.channels,), torch.float32, self.unit_state),
                StateNeed((self.conv_taps - 1, self.channels), torch.float32, self.conv_state))

    def takes_tensor_memory_tiles(self, page_size: int) -> bool:
        return True                  # no attention over pages: any cutting of a step into tiles will do

    # ---------------------------------------------------------------- running
    def forward(self, x, ctx, run: int):
        c = self.channels
        projected = linear(x, self.in_weight)
        entries = dict(row_starts=ctx.row_starts, state_slots=ctx.state_slots, token_row=ctx.token_row)
        u = kernels.short_convolution(projected[:, :c], self.conv_by_tap, bias=self.conv_bias, act=None,
                                      in_bias=self.x_bias, state=ctx.storage.state_of(run, self.conv_state), **entries)
        single = ctx.num_tokens == ctx.num_rows               # a step of single tokens
        fused = single and kernels.recurrent_unit_step_takes(ctx.num_rows, self.size)
        mixed = kernels.recurrent_unit(
            u, projected[:, c:2 * c], blocks=self.blocks, decay=self.decay, bias_r=self.r_bias, bias_i=self.i_bias,
            bias_y=self.y_bias, act=self.activation, state=ctx.storage.state_of(run, self.unit_state), single=single,
            pre=None if fused else kernels.block_products(u, self.gate_weight),
            weight=self.gate_weight if fused else None, **entries)
        return linear(mixed, self.o_weight, out_dtype=self.out_dtype)


register_part("mixer", "linear_recurrent_unit", LinearRecurrentUnit)
