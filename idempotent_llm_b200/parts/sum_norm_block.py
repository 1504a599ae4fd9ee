"""A block whose norms take the stream and a sublayer's output together:

    h <- N1(alpha h + mixer(h))
    h <- N2(alpha h + feed_forward(h))      if the layer has a feed-forward

The sublayers read the stream itself (in the storage dtype for their matrix products); the stream stays 32-bit.  One
kernel per sublayer makes the sum, norms it in groups, replaces the stream by it and writes it in the storage dtype for
whoever reads it next: the feed-forward, or the next layer's mixer, to which it is handed on as a ``CastStream``.
"""

from __future__ import annotations

from .base import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, Block, CastStream, NormedDelta
from .norm import GroupedRMSNorm


@BLOCKS.register("sum_norm")
class SumNormBlock(Block):
    reads_stream = True                 # its first sublayer reads the stream in the storage dtype (``CastStream``)

    @classmethod
    def declare(cls, spec, prefix=None):
        p = spec.prefix
        d = MIXERS.get(spec.mixer.kind).declare(spec.mixer, p) + NORMS.get(spec.mixer_norm.kind).declare(spec.mixer_norm, p)
        if spec.feed_forward is not None:
            d += FEED_FORWARDS.get(spec.feed_forward.kind).declare(spec.feed_forward, p)
            d += NORMS.get(spec.feed_forward_norm.kind).declare(spec.feed_forward_norm, p)
        return d

    def __init__(self, spec, weights, prefix, rt):
        p = spec.prefix
        self.spec, self.rt = spec, rt
        self.mixer = MIXERS.get(spec.mixer.kind)(spec.mixer, weights, p, rt)
        self.mixer_norm = NORMS.get(spec.mixer_norm.kind)(spec.mixer_norm, weights, p, rt)
        self.feed_forward = self.feed_forward_norm = None
        if spec.feed_forward is not None:
            self.feed_forward = FEED_FORWARDS.get(spec.feed_forward.kind)(spec.feed_forward, weights, p, rt)
            self.feed_forward_norm = NORMS.get(spec.feed_forward_norm.kind)(spec.feed_forward_norm, weights, p, rt)
        for n in (self.mixer_norm, self.feed_forward_norm):
            if n is not None and not isinstance(n, GroupedRMSNorm):
                raise ValueError("a layer that norms the sum has RMS norms in groups (its kernel adds and norms in one pass)")

    def _sum(self, h, y, norm):
        """``h <- norm(alpha h + y)`` in place; returns the stream in the storage dtype."""
        return self.rt.kernels.sum_norm(h, y, self.spec.alpha, norm.weight, norm.spec.eps, norm.spec.groups)

    def forward(self, h, pending, ctx, kv, state, writes_cache: bool):
        if isinstance(pending, CastStream):
            x = pending.x
        else:                                     # behind the embedding or a block of another kind: add what it left, then cast
            if isinstance(pending, NormedDelta):
                pending.add_into(h, self.rt.kernels)
            elif pending is not None:
                h += pending.sum(dim=0)
            x = h.to(self.rt.dtype)
        x = self._sum(h, self.mixer.forward(x, ctx, kv, state, writes_cache), self.mixer_norm)
        if self.feed_forward is not None:
            x = self._sum(h, self.feed_forward.forward(x, ctx), self.feed_forward_norm)
        return h, CastStream(x)
