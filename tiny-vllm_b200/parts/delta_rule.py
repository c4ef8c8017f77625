"""The gated delta rule: linear attention whose state corrects what it holds under a key before it writes.

q = W_q h and k = W_k h (``num_key_heads`` heads of ``key_dim``), v = W_v h (``num_heads`` heads of ``value_dim``; head h
uses q/k head h // (num_heads / num_key_heads)), each through a causal convolution over the last ``taps`` tokens, a
channel by itself, with SiLU behind it; q and k are then unit vectors over a head (``unit_eps`` beside the sum of
squares), q times ``query_scale``.  beta = sigmoid(W_b h) and g = exp(-exp(A_log) softplus(W_a h + dt_bias)), one number a
head.  Per head and request a float32 state S [key_dim, value_dim] runs along the tokens: S <- g S, u = beta (v - S^T k),
S <- S + k u^T, o = S^T q.  Every head's o is divided by its root mean square (``eps`` inside the root) and multiplied by
one weight for all heads (``out_norm``: "weight", "unit" for no weight, None for no norm), the concatenated heads are
multiplied by act(W_g h) (``gate``: "silu", "sigmoid" or None) and projected by W_o.

The mixer's memory is the state and the convolutions' last inputs, a slot a request each in the cache storage's state
arenas.  Unit vectors, decays, step sizes, state and sums are float32 whatever the storage type.
"""

from __future__ import annotations

import torch

from ..ops import kernels, linear
from .base import BuildContext, ParamSpec, Part, StateNeed
from .registry import register_part


class GatedDeltaRule(Part):
    def __init__(self, ctx: BuildContext, *, hidden_size: int, num_heads: int, num_key_heads: int, key_dim: int,
                 value_dim: int, taps: int, query_scale: float | None = None, unit_eps: float = 1e-6,
                 out_norm: str | None = "weight", eps: float = 0.0, gate: str | None = "silu",
                 float32_output: bool = False, names: dict | None = None) -> None:
        if num_key_heads <= 0 or num_heads % num_key_heads:
            raise ValueError("value heads must be a multiple of key heads")
        if not 0 < key_dim <= kernels.DELTA_MAX_DIM or value_dim <= 0:
            raise ValueError(f"the delta rule takes key sizes up to {kernels.DELTA_MAX_DIM}, not {key_dim}")
        if not 0 < taps <= kernels.CONV_TAPS[-1]:
            raise ValueError(f"the convolution takes up to {kernels.CONV_TAPS[-1]} taps, not {taps}")
        if out_norm not in (None, "unit", "weight"):
            raise ValueError(f"out_norm is None, 'unit' or 'weight', not {out_norm!r}")
        if gate not in kernels.RETENTION_ACTS:
            raise ValueError(f"gate is 'silu', 'sigmoid' or None, not {gate!r}")
        self.hidden_size, self.num_heads, self.num_key_heads = hidden_size, num_heads, num_key_heads
        self.key_dim, self.value_dim, self.taps = key_dim, value_dim, taps
        self.query_scale = float(key_dim) ** -0.5 if query_scale is None else float(query_scale)
        self.unit_eps, self.out_norm, self.eps, self.gate = float(unit_eps), out_norm, float(eps), gate
        self.out_dtype = torch.float32 if float32_output else None
        n = {"q": "q", "k": "k", "v": "v", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv", "b": "b", "a": "a",
             "a_log": "A_log", "dt_bias": "dt_bias", "g": "g", "norm": "norm", "o": "o", **(names or {})}
        self.names = {key: f"{ctx.prefix}.{value}" for key, value in n.items()}
        self.delta_state, self.conv_state = f"{ctx.prefix}.delta", f"{ctx.prefix}.conv"
        self.conv_taps = next(k for k in kernels.CONV_TAPS if k >= taps)
        self.in_weight = self.o_weight = self.conv_weight = self.a_log = self.dt_bias = self.norm_weight = None
        self.conv_by_tap = self.rate = None

    # ------------------------------------------------------------ declaration
    @property
    def key_cols(self) -> int:
        return self.num_key_heads * self.key_dim

    @property
    def out_cols(self) -> int:
        return self.num_heads * self.value_dim

    @property
    def conv_cols(self) -> int:
        """Columns [q | k | v], which the convolution runs over."""
        return 2 * self.key_cols + self.out_cols

    def param_specs(self):
        n, width, heads = self.names, self.hidden_size, self.num_heads
        rows = [(n["q"], self.key_cols), (n["k"], self.key_cols), (n["v"], self.out_cols)]
        if self.gate is not None:
            rows.append((n["g"], self.out_cols))
        rows += [(n["b"], heads), (n["a"], heads)]
        taps = ParamSpec.packed("conv_weight", [(n["q_conv"], self.key_cols), (n["k_conv"], self.key_cols),
                                                (n["v_conv"], self.out_cols)], self.taps)
        specs = [ParamSpec.packed("in_weight", rows, width),
                 ParamSpec(taps.attr, taps.shape, taps.sources, "vector", "unit_interval"),
                 ParamSpec.single("a_log", n["a_log"], (heads,), role="vector", init="unit_interval"),
                 ParamSpec.single("dt_bias", n["dt_bias"], (heads,), role="vector"),
                 ParamSpec.single("o_weight", n["o"], (width, self.out_cols))]
        if self.out_norm == "weight":
            specs.append(ParamSpec.single("norm_weight", n["norm"], (self.value_dim,), role="vector", init="around_one"))
        return specs

    def finalize(self) -> None:
        """What the kernels read: taps by age with the missing older ones as zeros, the rates -exp(A_log), both in
        float32, and the input projection with rows of zeros up to a multiple of 8, as the products want it."""
        if self.conv_by_tap is not None or self.conv_weight is None:
            return
        f32 = torch.float32
        self.conv_by_tap = torch.zeros((self.conv_taps, self.conv_cols), dtype=f32, device=self.conv_weight.device)
        self.conv_by_tap[self.conv_taps - self.taps:] = self.conv_weight.to(f32).t()
        self.rate = -torch.exp(self.a_log.to(f32)).contiguous()
        self.dt_bias = self.dt_bias.to(f32).contiguous()
        if self.norm_weight is not None:
            self.norm_weight = self.norm_weight.to(f32).contiguous()
        rows = self.in_weight.shape[0]
        if rows % 8:
            wide = torch.zeros((-(-rows // 8) * 8, self.hidden_size), dtype=self.in_weight.dtype, device=self.in_weight.device)
            wide[:rows] = self.in_weight
            self.in_weight = wide
        self.conv_weight = self.a_log = None

    def streamed_weights(self):
        return [self.in_weight, self.o_weight]

    def cache_need(self):
        return (StateNeed((self.num_heads, self.key_dim, self.value_dim), torch.float32, self.delta_state),
                StateNeed((self.conv_taps - 1, self.conv_cols), torch.float32, self.conv_state))

    def takes_tensor_memory_tiles(self, page_size: int) -> bool:
        return True                  # no attention over pages: any cutting of a step into tiles will do

    # ---------------------------------------------------------------- running
    def forward(self, x, ctx, run: int):
        projected = linear(x, self.in_weight)
        entries = dict(row_starts=ctx.row_starts, state_slots=ctx.state_slots, token_row=ctx.token_row)
        mixed = kernels.short_convolution(projected[:, :self.conv_cols], self.conv_by_tap, bias=None, act="silu",
                                          state=ctx.storage.state_of(run, self.conv_state), **entries)
        beta_at = self.conv_cols + (0 if self.gate is None else self.out_cols)
        gated = kernels.delta_rule(
            mixed, projected, q_at=0, k_at=self.key_cols, v_at=2 * self.key_cols, beta_at=beta_at,
            decay_at=beta_at + self.num_heads, heads=self.num_heads, key_heads=self.num_key_heads, dim=self.key_dim,
            vdim=self.value_dim, rate=self.rate, dt_bias=self.dt_bias, query_scale=self.query_scale,
            unit_eps=self.unit_eps, unit_norm=self.out_norm is not None, norm_weight=self.norm_weight, eps=self.eps,
            gate_at=None if self.gate is None else self.conv_cols, gate_act=self.gate,
            state=ctx.storage.state_of(run, self.delta_state), **entries)
        return linear(gated, self.o_weight, out_dtype=self.out_dtype)


register_part("mixer", "gated_delta_rule", GatedDeltaRule)
