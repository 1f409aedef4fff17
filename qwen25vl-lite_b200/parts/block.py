"""Pre-norm residual arrangement (reference src/qwen25vl_lite/text.py:196-206):
``x += mixer(norm1(x)); x += ffn(norm2(x))``.

The additions never run as kernels of their own.  A part that says ``accepts_residual``
adds its result into the float32 stream in the epilogue of its last product; otherwise the
result is carried as a pending update into the next norm kernel, which adds it before
normalising.  A part that says ``accepts_deferred_norm`` may be handed a norm that has not
run yet, to be computed inside its first product."""

from __future__ import annotations

from .base import Block, PendingUpdate, register_block


@register_block("prenorm_residual")
class PreNormResidualBlock(Block):
    def forward(self, ctx, x, pending, stop):
        mixer, ffn = self.mixer, self.feed_forward
        h = self.norms[0].forward(ctx, x, pending, defer=mixer.accepts_deferred_norm)
        if mixer.accepts_residual:
            mixed = mixer.forward(ctx, h, stop, residual=x)
        else:
            mixed = mixer.forward(ctx, h, stop)
        if ffn is None:                  # a layer of a mixer alone: its update is added by whoever normalises next
            return mixed
        h = self.norms[1].forward(ctx, x, mixed, defer=ffn.accepts_deferred_norm)
        if ffn.accepts_residual:
            return ffn.forward(ctx, h, residual=x)
        return ffn.forward(ctx, h)


@register_block("sandwich_residual")
class SandwichResidualBlock(Block):
    """Every sublayer is normalised before and after: ``x += norm1b(mixer(norm1(x)))``, then
    ``x += norm2b(ffn(norm2(x)))``; the norms come in that order (norm1, norm1b, norm2, norm2b).  A
    layer without a feed-forward has the mixer's two norms only.  The norm after a sublayer runs
    inside the kernel that adds the sublayer's result and normalises for the next one: the block
    hands its last result on as a ``PendingUpdate``."""

    def forward(self, ctx, x, pending, stop):
        h = self.norms[0].forward(ctx, x, pending)
        mixed = PendingUpdate(self.mixer.forward(ctx, h, stop), self.norms[1])
        if self.feed_forward is None:
            return mixed
        h = self.norms[2].forward(ctx, x, mixed)
        return PendingUpdate(self.feed_forward.forward(ctx, h), self.norms[3])


@register_block("scaled_residual")
class ScaledResidualBlock(Block):
    """Pre-norm sublayers whose results are scaled per channel on their way into the stream: ``x += s1 * mixer(norm1(x))``,
    then ``x += s2 * ffn(norm2(x))``; the norms come in that order (norm1, s1, norm2, s2, the scales being
    ``channel_scale`` parts).  A part that says ``accepts_scaled_residual`` is handed the stream and the scale and may add
    its result itself; otherwise the result is a ``PendingUpdate`` that the next norm's kernel scales and adds."""

    @staticmethod
    def _update(part, scale, x, *args):
        if not part.accepts_scaled_residual:
            return PendingUpdate(part.forward(*args), scale)
        value = part.forward(*args, residual=x, residual_scale=scale.weight)
        return None if value is None else PendingUpdate(value, scale)

    def forward(self, ctx, x, pending, stop):
        mixer, ffn = self.mixer, self.feed_forward
        h = self.norms[0].forward(ctx, x, pending, defer=mixer.accepts_deferred_norm)
        mixed = self._update(mixer, self.norms[1], x, ctx, h, stop)
        if ffn is None:
            return mixed
        h = self.norms[2].forward(ctx, x, mixed, defer=ffn.accepts_deferred_norm)
        return self._update(ffn, self.norms[3], x, ctx, h)


@register_block("hyper_residual")
class HyperResidualBlock(Block):
    """Pre-norm sublayers over a stream of several rows per token (``parts.norm.HyperRMSNorm``): each sublayer's norm reads
    the weighted sum of the rows, and its result is handed on as a ``PendingUpdate`` which the next norm's kernel writes
    into all rows with that sublayer's connection.  A layer without a feed-forward has the mixer's norm only at work."""

    def forward(self, ctx, x, pending, stop):
        mixed = PendingUpdate(self.mixer.forward(ctx, self.norms[0].forward(ctx, x, pending), stop), self.norms[0])
        if self.feed_forward is None:
            return mixed
        return PendingUpdate(self.feed_forward.forward(ctx, self.norms[1].forward(ctx, x, mixed)), self.norms[1])
