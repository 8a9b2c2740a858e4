"""The matrix memory of xLSTM (Beck et al., "xLSTM: Extended Long Short-Term Memory"): a recurrent mixer whose state is one
matrix per head, written through exponential gates and read through a normaliser.

Per head with dk key and dv value channels, h the mixer's input:

    q = W_q h dk^-1/2,  k = W_k h,  v = W_v h
    i = c tanh((W_i h + b_i) / c),  f = logsigmoid(c tanh((W_f h + b_f) / c))        one number per head, c = gate_cap
    m_t = max(f + m_(t-1), i)                                                         from m = 0
    S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k v^T,   n alike with k alone
    o = S^T q / (max(|n . q|, exp(-m)) + 1e-6)

Each head's o is divided by its root mean square; the joined heads are multiplied by a weight of all their channels and by
sigmoid(W_g h); W_o projects back.  q, k, v, the gate and both gates of the recurrence are one product over stacked weights;
what follows is float32.  n is one more value channel of the state whose value is always 1; m is kept beside it.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..cache.spec import FixedStateSpec
from ..weights.spec import MATRIX, NORM, VECTOR, WeightSpec
from .base import Mixer, StepContext, register

_NAMES = dict(q="q", k="k", v="v", gate="g", gate_in="i", gate_in_bias="i.b", gate_keep="f", gate_keep_bias="f.b", norm="norm", out="o")
DIVISOR_EPS = 1e-6


@register("mixer", "matrix_memory")
class MatrixMemory(Mixer):
    takes_lazy_input = True       # x goes to one product only
    writes_through_linear = True  # out is the out of the last product

    def __init__(self, hidden_size: int, num_heads: int, key_dim: int, value_dim: int, gate_cap: float, norm_eps: float,
                 names: Optional[dict] = None):
        if gate_cap <= 0:
            raise ValueError("gate_cap must be positive")
        self.hidden_size, self.num_heads, self.key_dim, self.value_dim = hidden_size, num_heads, key_dim, value_dim
        self.gate_cap, self.norm_eps = float(gate_cap), float(norm_eps)
        self.names = dict(_NAMES, **(names or {}))
        self.k_width, self.v_width = num_heads * key_dim, num_heads * value_dim
        self.inner_width = self.v_width
        self.stored_width = 2 * self.k_width + 2 * self.v_width + 2 * num_heads
        self.input_width = -(-self.stored_width // 8) * 8         # (zero rows behind the weights: whole 16-byte pieces)
        self.q_scale = float(key_dim) ** -0.5
        self.w_in = self.w_o = self.norm_w = self.bias_in = self.bias_keep = None

    def cache_specs(self):
        return [FixedStateSpec((self.num_heads, self.value_dim + 1, self.key_dim), torch.float32),
                FixedStateSpec((self.num_heads, self.value_dim + 1), torch.float32)]

    def weight_specs(self, prefix: str) -> list[WeightSpec]:
        n, W, H = self.names, self.hidden_size, self.num_heads
        return [WeightSpec(prefix + n["q"], (self.k_width, W), MATRIX),
                WeightSpec(prefix + n["k"], (self.k_width, W), MATRIX),
                WeightSpec(prefix + n["v"], (self.v_width, W), MATRIX),
                WeightSpec(prefix + n["gate"], (self.v_width, W), MATRIX),
                WeightSpec(prefix + n["gate_in"], (H, W), MATRIX),
                WeightSpec(prefix + n["gate_in_bias"], (H,), VECTOR),
                WeightSpec(prefix + n["gate_keep"], (H, W), MATRIX),
                WeightSpec(prefix + n["gate_keep_bias"], (H,), VECTOR),
                WeightSpec(prefix + n["norm"], (self.v_width,), NORM),
                WeightSpec(prefix + n["out"], (W, self.v_width), MATRIX)]

    def load(self, prefix, source, dtype, device) -> None:
        n = self.names
        rows = [source.get(prefix + n[x]) for x in ("q", "k", "v", "gate", "gate_in", "gate_keep")]
        rows.append(rows[0].new_zeros((self.input_width - self.stored_width, self.hidden_size)))
        self.w_in = ops.prepare_matrix(torch.cat(rows, dim=0).to(dtype).to(device))

        def f32(name):
            return source.get(prefix + n[name]).to(torch.float32).to(device).contiguous()
        self.bias_in, self.bias_keep, self.norm_w = f32("gate_in_bias"), f32("gate_keep_bias"), f32("norm")
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
        T, H, dk, dv = ctx.num_tokens, self.num_heads, self.key_dim, self.value_dim
        kw, vw = self.k_width, self.v_width
        state, maxima = cache
        at = 2 * kw + 2 * vw
        o = ctx.arena.alloc((T, vw), torch.float32)
        divisor = ctx.arena.alloc((T, H), torch.float32)
        ops.matrix_memory_scan(proj[:, :kw], proj[:, kw:2 * kw], proj[:, 2 * kw:2 * kw + vw], proj[:, at:at + H], proj[:, at + H:at + 2 * H],
                               self.bias_in, self.bias_keep, self.gate_cap, state, maxima, ctx, o, divisor, self.q_scale, DIVISOR_EPS,
                               H, dk, dv, write_state=write_cache)
        ops.group_norm_gate(o, proj[:, 2 * kw + vw:at], self.norm_w, self.norm_eps, H, inner, gate_kind="sigmoid", divisor=divisor, scale=scale)

    def forward(self, ctx: StepContext, x, cache, group, out, write_cache: bool = True) -> None:
        inner = ctx.arena.alloc((ctx.num_tokens, self.inner_width), ctx.dtype)
        self.mix_into(ctx, x, cache, group, inner, write_cache)
        ops.linear(inner, self.w_o, out)
