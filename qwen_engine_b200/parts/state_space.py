"""Mamba-2 (Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State
Space Duality"): a state-space mixer with one decay per head and token.

With H heads of P channels (inner = H P), a state of N channels and G groups of input and output maps:

    [z | x | B | C | dt] = W_in h                       inner, inner, G N, G N, H columns
    x, B, C = silu(conv([x | B | C]) + b_conv)          a causal convolution over `taps` tokens on each channel
    d = softplus(dt + dt_bias)
    S_t = exp(-exp(A_log) d_t) S_(t-1) + d_t B_t x_t^T   per head (head i reads group i // (H / G)); S: N x P, zero at first
    y_t = S_t^T C_t + D x_t
    y <- rms-normed in `norm_groups` equal parts of (y * silu(z)), times the norm's weight;  W_out y

The projection is one product (its rows padded with zero rows to whole 16-byte pieces); the convolution with bias and silu
is one kernel, the recurrence with its step sizes and decays another, gate and norm a third.  S, d, the decays and the norm
are float32.  Two states of fixed size per request: S, and the convolution's last taps - 1 inputs.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..cache.spec import FixedStateSpec
from ..weights.spec import MATRIX, NORM, TAPS, VECTOR, WeightSpec
from .base import Mixer, StepContext, register

_NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "rate": "A_log", "skip": "D", "norm": "norm", "out": "o"}


@register("mixer", "state_space")
class StateSpace(Mixer):
    takes_lazy_input = True       # x goes to one product only
    writes_through_linear = True  # out is the out of the last product

    def __init__(self, hidden_size: int, num_heads: int, value_dim: int, state_dim: int, num_groups: int, conv_taps: int,
                 norm_groups: int, norm_eps: float, names: Optional[dict] = None):
        if num_heads % num_groups:
            raise ValueError("num_heads must be a multiple of num_groups")
        if (num_heads * value_dim) % norm_groups:
            raise ValueError(f"{num_heads * value_dim} channels do not split into {norm_groups} equal parts")
        if conv_taps < 1:
            raise ValueError("conv_taps must be positive")
        self.hidden_size, self.num_heads, self.value_dim, self.state_dim = hidden_size, num_heads, value_dim, state_dim
        self.num_groups, self.conv_taps, self.norm_groups, self.norm_eps = num_groups, conv_taps, norm_groups, float(norm_eps)
        self.names = dict(_NAMES, **(names or {}))
        self.inner = num_heads * value_dim
        self.map_width = num_groups * state_dim
        self.conv_width = self.inner + 2 * self.map_width
        self.stored_width = self.inner + self.conv_width + num_heads
        self.inner_width = self.inner
        self.input_width = -(-self.stored_width // 8) * 8
        self.w_in = self.w_conv = self.conv_bias = self.dt_bias = self.log_rate = self.skip = self.norm_w = self.w_o = None

    def cache_specs(self):
        # the recurrence's state (a channel's state channels side by side), and the convolution's last inputs
        specs = [FixedStateSpec((self.num_heads, self.value_dim, self.state_dim), torch.float32)]
        if self.conv_taps > 1:
            specs.append(FixedStateSpec((self.conv_taps - 1, self.conv_width), torch.float32))
        return specs

    def weight_specs(self, prefix: str) -> list[WeightSpec]:
        n, W, H = self.names, self.hidden_size, self.num_heads
        return [WeightSpec(prefix + n["in"], (self.stored_width, W), MATRIX),
                WeightSpec(prefix + n["conv"], (self.conv_width, self.conv_taps), TAPS),
                WeightSpec(prefix + n["conv_bias"], (self.conv_width,), VECTOR),
                WeightSpec(prefix + n["dt_bias"], (H,), VECTOR),
                WeightSpec(prefix + n["rate"], (H,), VECTOR),
                WeightSpec(prefix + n["skip"], (H,), VECTOR),
                WeightSpec(prefix + n["norm"], (self.inner,), NORM),
                WeightSpec(prefix + n["out"], (W, self.inner), MATRIX)]

    def load(self, prefix, source, dtype, device) -> None:
        n = self.names

        def f32(name):
            return source.get(prefix + n[name]).to(torch.float32).to(device).contiguous()
        w = source.get(prefix + n["in"])
        w = torch.cat([w, w.new_zeros((self.input_width - self.stored_width, w.shape[1]))], dim=0)
        self.w_in = ops.prepare_matrix(w.to(dtype).to(device))
        self.w_conv = source.get(prefix + n["conv"]).to(torch.float32).t().contiguous().to(device)        # [taps, channels]
        self.conv_bias, self.dt_bias, self.log_rate = f32("conv_bias"), f32("dt_bias"), f32("rate")
        self.skip, self.norm_w = f32("skip"), f32("norm")
        self.w_o = ops.prepare_matrix(source.get(prefix + n["out"]).to(dtype).to(device))

    def first_weights(self):
        return self.w_in

    def output_weight(self):
        return self.w_o

    def input_weight(self):
        return self.w_in

    def mix_into(self, ctx: StepContext, x, cache, group, inner, write_cache: bool = True, scale: float = 1.0) -> None:
        proj = ctx.arena.alloc((ctx.num_tokens, self.input_width), ctx.dtype)
        ops.linear(x, self.w_in, proj)
        self.mix_projected(ctx, proj, cache, group, inner, write_cache, scale)

    def mix_projected(self, ctx: StepContext, proj, cache, group, inner, write_cache: bool = True, scale: float = 1.0) -> None:
        T, n, C, GN, H = ctx.num_tokens, self.inner, self.conv_width, self.map_width, self.num_heads
        state, conv_state = cache if isinstance(cache, tuple) else (cache, None)
        xbc = ctx.arena.alloc((T, C), ctx.dtype)
        ops.conv_act(proj[:, n:n + C], self.w_conv, conv_state, ctx, xbc, out_bias=self.conv_bias, silu=True, write_state=write_cache)
        y = ctx.arena.alloc((T, n), torch.float32)
        ops.state_space_scan(xbc[:, :n], xbc[:, n:n + GN], xbc[:, n + GN:], proj[:, n + C:n + C + H], self.dt_bias, self.log_rate, self.skip,
                             state, ctx, y, H, self.num_groups, self.state_dim, self.value_dim, write_state=write_cache)
        ops.group_norm_gate(y, proj[:, :n], self.norm_w, self.norm_eps, self.norm_groups, inner, gate_kind="silu", gate_first=True, scale=scale)

    def forward(self, ctx: StepContext, x, cache, group, out, write_cache: bool = True) -> None:
        inner = ctx.arena.alloc((ctx.num_tokens, self.inner_width), ctx.dtype)
        self.mix_into(ctx, x, cache, group, inner, write_cache)
        ops.linear(inner, self.w_o, out)
