"""A selective scan (Mamba): a state a channel whose step size, input and output directions come from the token.

[x | z] = W_in h, ``inner`` channels each.  x passes a causal convolution over the last ``taps`` tokens, a channel by
itself, with a bias and SiLU behind it.  W_x x = [low (``dt_rank``) | B (``state``) | C (``state``)], the step sizes
are dt = softplus(W_dt low + b), one a channel, and A = -exp(A_log).  Per request a float32 state S [inner, state]
runs along the tokens: S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n, y_c = sum_n S[c, n] C_n + D_c x_c; the
output is W_o (y * silu(z)).

The mixer's memory is the state and the convolution's last inputs, a slot a request each in the cache storage's
state arenas.  Step sizes, exponentials, state and sums are float32 whatever the storage type.
"""

from __future__ import annotations

import torch

from ..ops import kernels, linear
from .base import BuildContext, ParamSpec, Part, StateNeed
from .registry import register_part


class SelectiveScan(Part):
    """``hosted=True``: a block (or a mixer of mixers) computes the projections from and to the model width; the part
    then names its share (``input_rows``, ``output_cols``) and works between the two products (``between``)."""

    def __init__(self, ctx: BuildContext, *, hidden_size: int, inner: int, state: int, dt_rank: int, taps: int,
                 hosted: bool = False, float32_output: bool = False, names: dict | None = None) -> None:
        if not 0 < state <= kernels.SCAN_MAX_STATE:
            raise ValueError(f"the scan takes states of up to {kernels.SCAN_MAX_STATE} numbers a channel, not {state}")
        if not 0 < taps <= kernels.CONV_TAPS[-1]:
            raise ValueError(f"the convolution takes up to {kernels.CONV_TAPS[-1]} taps, not {taps}")
        self.hidden_size, self.inner, self.state, self.dt_rank, self.taps = hidden_size, inner, state, dt_rank, taps
        self.hosted = hosted
        self.out_dtype = torch.float32 if float32_output else None
        n = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "x": "x", "dt": "dt", "dt_bias": "dt.b",
             "a_log": "A_log", "d": "D", "o": "o", **(names or {})}
        self.names = {key: f"{ctx.prefix}.{value}" for key, value in n.items()}
        self.scan_state, self.conv_state = f"{ctx.prefix}.scan", f"{ctx.prefix}.conv"
        # sizes the products want: the low-rank part and the whole row in steps of 8, zeros in between
        self.rank_cols = -(-dt_rank // 8) * 8
        self.x_cols = -(-(self.rank_cols + 2 * state) // 8) * 8
        self.conv_taps = next(k for k in kernels.CONV_TAPS if k >= taps)
        self.in_weight = self.o_weight = self.conv_weight = self.conv_bias = self.x_weight = self.dt_weight = None
        self.dt_bias = self.a_log = self.d = self.a = self.conv_by_tap = None

    # ------------------------------------------------------------ declaration
    def input_rows(self):
        return [(self.names["in"], 2 * self.inner)]

    def output_cols(self):
        return (self.names["o"], self.inner)

    def param_specs(self):
        n, inner = self.names, self.inner
        specs = []
        if not self.hosted:
            specs += [ParamSpec.packed("in_weight", self.input_rows(), self.hidden_size),
                      ParamSpec.single("o_weight", n["o"], (self.hidden_size, inner))]
        return specs + [
            ParamSpec.single("conv_weight", n["conv"], (inner, self.taps), role="vector", init="unit_interval"),
            ParamSpec.single("conv_bias", n["conv_bias"], (inner,), role="vector"),
            ParamSpec.single("x_weight", n["x"], (self.dt_rank + 2 * self.state, inner)),
            ParamSpec.single("dt_weight", n["dt"], (inner, self.dt_rank)),
            ParamSpec.single("dt_bias", n["dt_bias"], (inner,), role="vector"),
            ParamSpec.single("a_log", n["a_log"], (inner, self.state), role="vector"),
            ParamSpec.single("d", n["d"], (inner,), role="vector", init="around_one")]

    def finalize(self) -> None:
        """What the kernels read: taps by age with the missing older ones as zeros, A itself, both in float32, and
        the two small products' weights with their low-rank part widened by zeros."""
        if self.conv_by_tap is not None:
            return
        f32 = torch.float32
        self.conv_by_tap = torch.zeros((self.conv_taps, self.inner), dtype=f32, device=self.conv_weight.device)
        self.conv_by_tap[self.conv_taps - self.taps:] = self.conv_weight.to(f32).t()
        self.a = -torch.exp(self.a_log.to(f32)).contiguous()
        self.conv_bias, self.dt_bias, self.d = (t.to(f32).contiguous() for t in (self.conv_bias, self.dt_bias, self.d))
        rank, state = self.dt_rank, self.state
        widened = torch.zeros((self.x_cols, self.inner), dtype=self.x_weight.dtype, device=self.x_weight.device)
        widened[:rank] = self.x_weight[:rank]
        widened[self.rank_cols:self.rank_cols + 2 * state] = self.x_weight[rank:]
        self.x_weight = widened
        widened = torch.zeros((self.inner, self.rank_cols), dtype=self.dt_weight.dtype, device=self.dt_weight.device)
        widened[:, :rank] = self.dt_weight
        self.dt_weight = widened
        self.conv_weight = self.a_log = None

    def streamed_weights(self):
        return [] if self.hosted else [self.in_weight, self.o_weight]

    def cache_need(self):
        return (StateNeed((self.inner, self.state), torch.float32, self.scan_state),
                StateNeed((self.conv_taps - 1, self.inner), torch.float32, self.conv_state))

    def takes_tensor_memory_tiles(self, page_size: int) -> bool:
        return True                  # no attention over pages: any cutting of a step into tiles will do

    # ---------------------------------------------------------------- running
    def between(self, projected, at: int, ctx, out, run: int) -> None:
        """From this mixer's columns [x | z] of a projection (from ``at`` on) to y * silu(z) in ``out``."""
        inner, rank = self.inner, self.rank_cols
        entries = dict(row_starts=ctx.row_starts, state_slots=ctx.state_slots, token_row=ctx.token_row)
        x = kernels.short_convolution(projected[:, at:at + inner], self.conv_by_tap, bias=self.conv_bias, act="silu",
                                      state=ctx.storage.state_of(run, self.conv_state), **entries)
        mixed = linear(x, self.x_weight)
        low = mixed[:, :rank]
        single = ctx.num_tokens == ctx.num_rows               # a step of single tokens
        fused = single and kernels.selective_step_takes(ctx.num_rows, rank)
        pre = None if fused else linear(low, self.dt_weight, out_dtype=torch.float32)
        kernels.selective_scan(
            x, pre=pre, low=low if fused else None, dt_weight=self.dt_weight if fused else None,
            z=projected[:, at + inner:at + 2 * inner], b=mixed[:, rank:rank + self.state],
            c=mixed[:, rank + self.state:rank + 2 * self.state], a=self.a, d=self.d, dt_bias=self.dt_bias,
            state=ctx.storage.state_of(run, self.scan_state), out=out, single=single, **entries)

    def forward(self, x, ctx, run: int):
        projected = linear(x, self.in_weight)
        inner = torch.empty((x.shape[0], self.inner), dtype=x.dtype, device=x.device)
        self.between(projected, 0, ctx, inner, run)
        return linear(inner, self.o_weight, out_dtype=self.out_dtype)


register_part("mixer", "selective_scan", SelectiveScan)
