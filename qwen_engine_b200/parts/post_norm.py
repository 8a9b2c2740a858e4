"""A residual block whose sublayers read the stream itself and norm what they return.

For the float32 stream x of a layer, with a sublayer f (the mixer, then the feed-forward):

    x <- x + norm(f(x))

In bfloat16 a sublayer reads x rounded once to the compute type: the kernel that writes x (the embedding, or the add of
the sublayer before) leaves that copy beside the stream (``ops.ResidualStream.copy``), so no kernel only rounds.  In
float32 it reads the stream as it is.  Norm and add are one pass over a row.
"""
from __future__ import annotations

from typing import Optional

from .base import Block, PartSpec, StepContext, register


@register("block", "post_norm")
class PostNormBlock(Block):
    keeps_copy = True

    def __init__(self, hidden_size: int, mixer: PartSpec, feed_forward: Optional[PartSpec], norm: PartSpec,
                 mixer_prefix: str = "mix.", ffn_prefix: str = "mlp.", norm1_prefix: str = "norm1", norm2_prefix: str = "norm2"):
        self.hidden_size = hidden_size
        self.mixer = mixer.build("mixer")
        self.norm1 = norm.build("norm")
        self.ffn = feed_forward.build("feed_forward") if feed_forward is not None else None
        self.norm2 = norm.build("norm") if self.ffn is not None else None
        self.prefixes = (mixer_prefix, norm1_prefix, ffn_prefix, norm2_prefix)

    def _parts(self):
        return [(part, p) for part, p in zip((self.mixer, self.norm1, self.ffn, self.norm2), self.prefixes) if part is not None]

    @property
    def capturable(self) -> bool:
        return all(getattr(part, "capturable", True) for part, _ in self._parts())

    def weight_specs(self, prefix: str):
        return [s for part, p in self._parts() for s in part.weight_specs(prefix + p)]

    def load(self, prefix, source, dtype, device) -> None:
        for part, p in self._parts():
            part.load(prefix + p, source, dtype, device)

    def first_weights(self):
        return self.mixer.first_weights()

    def forward(self, ctx: StepContext, stream, cache, group, write_cache) -> None:
        if stream.has_delta:
            raise RuntimeError("post_norm: the stream carries a branch output that nobody added")
        if getattr(ctx, "extras", None) is not None:
            ctx.extras["weights_after_mixer"] = self.ffn.first_weights() if self.ffn is not None else None
        mark = ctx.arena.mark()
        out = ctx.arena.alloc((ctx.num_tokens, self.hidden_size), ctx.dtype)
        self.mixer.forward(ctx, stream.rounded(), cache, group, out, write_cache)
        self._way_back(ctx, self.norm1, stream, out)
        ctx.arena.release(mark)
        if self.ffn is not None:
            out = ctx.arena.alloc((ctx.num_tokens, self.hidden_size), ctx.dtype)
            self.ffn.forward(ctx, stream.rounded(), out)
            self._way_back(ctx, self.norm2, stream, out)
            ctx.arena.release(mark)

    @staticmethod
    def _way_back(ctx, norm, stream, out) -> None:
        norm.norm_add(ctx, stream.resid, out, stream.resid, cast=stream.copy)
        stream.n_ssq, stream.copy_current = 0, stream.copy is not None
