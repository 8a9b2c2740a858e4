"""A residual block whose mixer and feed-forward run side by side, each behind a norm of its own of the same stream:

    x <- x + (mixer(norm1(x)) + ffn(norm2(x)))

Both norms divide by the same root mean square, so one pass over the stream makes both sublayers' inputs; the same pass
adds what the layer before left pending and the bias that the mixer's result carries (``Mixer.output_bias``).  The
sublayers' last products add into the stream where few rows allow it; otherwise both results stay pending
(``ResidualStream.delta`` and ``second``) for the pass that opens the next layer.  A layer may have no feed-forward."""
from __future__ import annotations

from typing import Optional

from .. import ops
from .base import Block, PartSpec, StepContext, register


@register("block", "side_by_side")
class SideBySideBlock(Block):
    takes_second = True
    adds_output_bias = True

    def __init__(self, hidden_size: int, mixer: PartSpec, feed_forward: Optional[PartSpec], norm: PartSpec,
                 mixer_prefix: str = "mix.", ffn_prefix: str = "mlp.", norm1_prefix: str = "norm1", norm2_prefix: str = "norm2"):
        self.hidden_size = hidden_size
        self.norm1 = norm.build("norm")
        self.norm2 = norm.build("norm") if feed_forward is not None else None
        if not hasattr(self.norm1, "normed_pair"):
            raise ValueError(f"side_by_side: norm {norm.name!r} does not make two norms in one pass")
        self.mixer = mixer.build("mixer")
        self.ffn = feed_forward.build("feed_forward") if feed_forward is not None else None
        self.prefixes = (norm1_prefix, mixer_prefix, norm2_prefix, ffn_prefix)

    def _parts(self):
        return [(part, p) for part, p in zip((self.norm1, self.mixer, self.norm2, self.ffn), self.prefixes) if part is not None]

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
        mark = ctx.arena.mark()
        h1, h2 = self.norm1.normed_pair(ctx, stream, self.norm2, bias=self.mixer.output_bias())
        self._run(ctx, stream, self.mixer, lambda out: self.mixer.forward(ctx, h1, cache, group, out, write_cache),
                  "weights_after_mixer", self.ffn)
        if self.ffn is not None:
            self._run(ctx, stream, self.ffn, lambda out: self.ffn.forward(ctx, h2, out), None, None)
        ctx.arena.release(mark)

    def _run(self, ctx, stream, part, run, hint, follows) -> None:
        """Run a sublayer: its result joins the stream at once, or stays pending in the buffer that is free."""
        if hint is not None and getattr(ctx, "extras", None) is not None:
            ctx.extras[hint] = follows.first_weights() if follows is not None else None
        if not stream.has_delta:
            out = ops.ResidualSink(stream) if part.writes_through_linear else stream.delta
            run(out)
            if not isinstance(out, ops.ResidualSink):
                stream.has_delta, stream.n_ssq = True, 0
            return
        run(stream.second_buffer(ctx.arena.alloc_step))
        stream.has_second, stream.n_ssq = True, 0
