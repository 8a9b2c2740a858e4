"""Latent attention: softmax attention whose keys and values are read out of one small latent per token.

For the mixer's input h, H heads with dn unrotated and dr rotated query/key channels and dv value channels, a latent
of R channels:

    c_q = rmsnorm(W_dq h),  q_h = W_uq,h c_q = [q_plain (dn) | q_rot (dr)]
    [c' | k_rot] = W_dkv h,  c = rmsnorm(c') (R channels),  k_rot (dr channels) is one key part for all heads
    k_plain,h = W_uk,h c,  v_h = W_uv,h c
    score_h(i, j) = scale (q_plain,h,i . k_plain,h,j + rot(q_rot,h,i) . rot(k_rot,j)),  j <= i,  softmax over j

The rotation turns the pairs (x[i], x[i + dims/2]) of the first ``dims`` rotated channels by position x base^(-2i/dims).
The joined heads are multiplied by sigmoid(W_g h) and projected by W_o.

Options (all off by default):

* ``query_rank`` None: the queries are projected from h directly, q_h = W_q,h h (one matrix, no query latent, no norm).
* ``pairing`` "interleaved": the pairs are (x[2i], x[2i + 1]).  The rotated rows of the query's matrix and of W_dkv are put
  into half-split order at load, which leaves every product of rotated parts as it was, so the kernels know one pairing.
* ``window``: the query at position i sees the keys at j > i - window only.  ``cache_window``: how many of the last keys the
  cache slot keeps where other layers with longer windows read it too (None: all of them; absent: ``window``).
* ``sink``: one stored number per head; exp(sink_h) joins head h's softmax denominator.
* ``output_gate`` "sigmoid_head": head h's output is multiplied by sigmoid(W_g h)_h, one number per head; formed where the
  heads' values are (the epilogue of the product with W_uv).
* ``shared_kv``: the layer has no W_dkv.  It reads the cache slot that another layer writes (the plan entry says
  ``write_cache`` False), with queries, W_uk, W_uv, window, sink and gate of its own.

The cache holds c and the rotated k_rot, one plane of R + dr channels per token and nothing per head.  W_uk is folded into the query
(q_lat,h = W_uk,h^T q_plain,h) and W_uv applied after the softmax, so the paged attention kernels see ONE key/value
head of R + dr channels whose values are the keys' first R channels, for prompt portions and decoded tokens alike.
Norms, angles, scores and softmax are float32.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..cache.spec import PagedKVSpec
from ..weights.spec import MATRIX, NORM, VECTOR, WeightSpec
from .base import Mixer, StepContext, register, step_hint

_NAMES = dict(q="q", q_down="dq", q_norm="dq.norm", q_up="uq", kv_down="dkv", kv_norm="dkv.norm", k_up="uk", v_up="uv",
              gate="g", out="o", sink="sink")
_SAME = object()


def _align8(n: int) -> int:
    return -(-n // 8) * 8


def _pad_rows_to(w: torch.Tensor, rows: int) -> torch.Tensor:
    """Zero rows behind the matrix's own (the columns of a stacked product then start on 16-byte boundaries)."""
    return w if w.shape[0] == rows else torch.cat([w, w.new_zeros((rows - w.shape[0], w.shape[1]))], dim=0)


@register("mixer", "latent_attention")
class LatentAttention(Mixer):
    takes_lazy_input = True       # x goes to one product only
    writes_through_linear = True  # out is the out of the last product

    def __init__(self, hidden_size: int, num_heads: int, plain_dim: int, rot_dim: int, value_dim: int, latent_dim: int,
                 query_rank: Optional[int], scale: float, norm_eps: float, rope_base: float, rope_dims: Optional[int] = None,
                 output_gate: Optional[str] = "sigmoid", names: Optional[dict] = None, pairing: str = "half",
                 window: Optional[int] = None, cache_window=_SAME, sink: bool = False, shared_kv: bool = False):
        if output_gate not in (None, "sigmoid", "sigmoid_head"):
            raise ValueError(f"unknown output gate {output_gate!r}")
        if pairing not in ("half", "interleaved"):
            raise ValueError(f"unknown pairing {pairing!r}")
        if window is not None and window < 1:
            raise ValueError("a window holds at least the token itself")
        self.pairing, self.window, self.sink, self.shared_kv = pairing, window, bool(sink), bool(shared_kv)
        self.cache_window = window if cache_window is _SAME else cache_window
        if self.cache_window is not None and (window is None or self.cache_window < window):
            raise ValueError(f"a cache of the last {self.cache_window} keys does not serve a window of {window}")
        self.hidden_size, self.num_heads = hidden_size, num_heads
        self.plain_dim, self.rot_dim, self.value_dim = plain_dim, rot_dim, value_dim
        self.latent_dim, self.query_rank = latent_dim, query_rank
        self.scale, self.norm_eps = float(scale), float(norm_eps)
        self.rope_base = float(rope_base)
        self.rope_dims = rot_dim if rope_dims is None else int(rope_dims)
        if self.rope_dims % 2 or not (0 <= self.rope_dims <= rot_dim):
            raise ValueError(f"rope_dims {self.rope_dims} must be even and within rot_dim {rot_dim}")
        self.output_gate = output_gate
        self.names = dict(_NAMES, **(names or {}))
        self.cache_dim = latent_dim + rot_dim                     # channels of a token's cache row
        self.q_width = num_heads * (plain_dim + rot_dim)
        self.inner_width = num_heads * value_dim
        # the stacked input product's columns: queries (or their latent), latent with the shared key part, gate
        self.lead_width = _align8(self.q_width) if query_rank is None else query_rank
        self.gate_width = 0 if not output_gate else self.inner_width if output_gate == "sigmoid" else _align8(num_heads)
        kv_width = 0 if shared_kv else _align8(self.cache_dim) if query_rank is None else self.cache_dim
        self.gate_at = self.lead_width + kv_width
        self.input_width = self.gate_at + self.gate_width
        self.w_in = self.w_uq = self.w_uk_t = self.w_uv = self.w_o = None
        self.q_norm_w = self.kv_norm_w = self.inv_freq = self.sinks = None

    def cache_spec(self):
        return PagedKVSpec(1, self.cache_dim, self.cache_window, planes=1)

    def attention_geometry(self):
        return (self.num_heads, 1, self.cache_dim, self.window or 0, False, 1)

    def weight_specs(self, prefix: str) -> list[WeightSpec]:
        n, H, W = self.names, self.num_heads, self.hidden_size
        if self.query_rank is None:
            specs = [WeightSpec(prefix + n["q"], (self.q_width, W), MATRIX)]
        else:
            specs = [WeightSpec(prefix + n["q_down"], (self.query_rank, W), MATRIX),
                     WeightSpec(prefix + n["q_norm"], (self.query_rank,), NORM),
                     WeightSpec(prefix + n["q_up"], (self.q_width, self.query_rank), MATRIX)]
        if not self.shared_kv:
            specs += [WeightSpec(prefix + n["kv_down"], (self.cache_dim, W), MATRIX),
                      WeightSpec(prefix + n["kv_norm"], (self.latent_dim,), NORM)]
        specs += [
            WeightSpec(prefix + n["k_up"], (H * self.plain_dim, self.latent_dim), MATRIX),
            WeightSpec(prefix + n["v_up"], (H * self.value_dim, self.latent_dim), MATRIX),
            WeightSpec(prefix + n["out"], (W, H * self.value_dim), MATRIX),
        ]
        if self.output_gate:
            specs.append(WeightSpec(prefix + n["gate"], (H if self.output_gate == "sigmoid_head" else H * self.value_dim, W), MATRIX))
        if self.sink:
            specs.append(WeightSpec(prefix + n["sink"], (H,), VECTOR))
        return specs

    def _rotated_rows(self, w: torch.Tensor, heads: int, plain: int) -> torch.Tensor:
        """The rows of a matrix whose outputs are, head by head, ``plain`` channels and then rot_dim rotated ones, with the
        rotated ones in the order the kernels turn them in."""
        if self.pairing == "half":
            return w
        d = self.rope_dims
        order = list(range(0, d, 2)) + list(range(1, d, 2)) + list(range(d, self.rot_dim))
        w = w.reshape(heads, plain + self.rot_dim, w.shape[1])
        return torch.cat([w[:, :plain], w[:, plain:][:, order]], dim=1).reshape(heads * (plain + self.rot_dim), w.shape[2])

    def load(self, prefix, source, dtype, device) -> None:
        n, H = self.names, self.num_heads
        q_up = self._rotated_rows(source.get(prefix + (n["q"] if self.query_rank is None else n["q_up"])), H, self.plain_dim)
        rows = [_pad_rows_to(q_up if self.query_rank is None else source.get(prefix + n["q_down"]), self.lead_width)]
        if not self.shared_kv:
            rows.append(_pad_rows_to(self._rotated_rows(source.get(prefix + n["kv_down"]), 1, self.latent_dim), self.gate_at - self.lead_width))
            self.kv_norm_w = source.get(prefix + n["kv_norm"]).to(torch.float32).to(device).contiguous()
        if self.output_gate:
            rows.append(_pad_rows_to(source.get(prefix + n["gate"]), self.gate_width))
        self.w_in = ops.prepare_matrix(torch.cat(rows, dim=0).to(dtype).to(device))
        if self.query_rank is not None:
            self.w_uq = ops.prepare_matrix(q_up.to(dtype).to(device))
            self.q_norm_w = source.get(prefix + n["q_norm"]).to(torch.float32).to(device).contiguous()
        if self.sink:
            self.sinks = source.get(prefix + n["sink"]).to(torch.float32).to(device).contiguous()
        # W_uk per head, transposed: the fold of a head's plain query into the latent's channels is a product with it
        uk = source.get(prefix + n["k_up"]).reshape(H, self.plain_dim, self.latent_dim)
        self.w_uk_t = uk.transpose(1, 2).contiguous().to(dtype).to(device)
        self.w_uv = source.get(prefix + n["v_up"]).reshape(H, self.value_dim, self.latent_dim).contiguous().to(dtype).to(device)
        self.w_o = ops.prepare_matrix(source.get(prefix + n["out"]).to(dtype).to(device))
        i = torch.arange(max(self.rope_dims // 2, 1), dtype=torch.float64)
        self.inv_freq = (self.rope_base ** (-2.0 * i / max(self.rope_dims, 1))).to(torch.float32).to(device).contiguous()

    def first_weights(self):
        return self.w_in

    def output_weight(self):
        return self.w_o

    def mix_into(self, ctx: StepContext, x, cache, group, inner, write_cache: bool = True, scale: float = 1.0) -> None:
        T, H = ctx.num_tokens, self.num_heads
        dn, dr, dv, R, D = self.plain_dim, self.rot_dim, self.value_dim, self.latent_dim, self.cache_dim
        view = ctx.groups[group]
        proj = ctx.arena.alloc((T, self.input_width), ctx.dtype)
        ops.linear(x, self.w_in, proj)
        if self.query_rank is None:
            q = proj[:, :self.q_width]
        else:
            cq = ctx.arena.alloc((T, self.query_rank), ctx.dtype)
            ops.head_norm_gate(proj[:, :self.query_rank], None, self.q_norm_w, self.norm_eps, cq, 1, self.query_rank, gate_kind=None)
            q = ctx.arena.alloc((T, self.q_width), ctx.dtype)
            ops.linear(cq, self.w_uq, q)
        writes = write_cache and not self.shared_kv
        down = None if self.shared_kv else proj[:, self.lead_width:self.lead_width + D]
        qlat = ctx.arena.alloc((T, H * D), ctx.dtype)
        ops.latent_prepare(down, q, self.kv_norm_w, self.norm_eps, ctx.positions, self.inv_freq, self.rope_dims, cache,
                           view.slot_mapping, qlat, H, dn, R, dr, write_kv=writes)
        ops.head_linear(q, self.w_uk_t, qlat, dn + dr, D)
        olat = ctx.arena.alloc((T, H * D), ctx.dtype)
        ops.paged_attention(qlat, cache, view.block_tables, ctx, olat, self.scale, self.window or 0, H, 1, D, sinks=self.sinks,
                            value_dim=R)
        gate = proj[:, self.gate_at:self.gate_at + (H if self.output_gate == "sigmoid_head" else self.gate_width)] if self.output_gate else None
        per_head = self.output_gate == "sigmoid_head"
        elementwise = self.output_gate == "sigmoid" or scale != 1.0
        attn = ctx.arena.alloc((T, H * dv), ctx.dtype) if elementwise or not inner.is_contiguous() else inner
        ops.head_linear(olat, self.w_uv, attn, D, dv, gate=gate if per_head else None)
        if attn is not inner:
            ops.head_norm_gate(attn, None if per_head else gate, None, 0.0, inner, H, dv,
                               gate_kind=None if per_head else self.output_gate, scale=scale)

    def forward(self, ctx: StepContext, x, cache, group, out, write_cache: bool = True) -> None:
        inner = ctx.arena.alloc((ctx.num_tokens, self.inner_width), ctx.dtype)
        if self.query_rank is None:
            ops.prefetch_next(self.w_o)              # (the product of a few rows asks L2 for the matrix the mixer ends with)
        self.mix_into(ctx, x, cache, group, inner, write_cache)
        ops.prefetch_next(step_hint(ctx, "weights_after_mixer"))
        ops.linear(inner, self.w_o, out)
        ops.prefetch_next(None)
