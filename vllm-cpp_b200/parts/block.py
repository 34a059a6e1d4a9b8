"""The pre-norm arrangement of a decoder layer:
x += mixer(norm1(x)); x += feed_forward(norm2(x))   (src/model.cpp:1181-1250).

The additions are not done here: each norm adds the delta still pending from the
part before it while it normalises, so the block hands its last delta on to
whatever norm comes next (the next layer's, or the final one)."""
from __future__ import annotations

from .base import Block


class PreNormBlock(Block):
    """parts: ``norm1``, ``mixer`` and, unless the layer has none, ``norm2`` and ``feed_forward``."""

    def __init__(self, params, prefix, build, parts):
        super().__init__(params, prefix, build, parts)
        if ("feed_forward" in parts) != ("norm2" in parts):
            raise ValueError("a feed-forward and its norm come together")

    def forward(self, resid, pending, ctx, cache, writes=True):
        mark = getattr(ctx, "mark", lambda label: None)     # kernel groups for the profile, where the step keeps one
        y = self.parts["norm1"].forward(resid, pending)
        d = self.parts["mixer"].forward(y, ctx, cache, writes)
        mark("mixer")
        if "feed_forward" not in self.parts:
            return d
        y = self.parts["norm2"].forward(resid, d)
        out = self.parts["feed_forward"].forward(y, ctx)
        mark("feed_forward")
        return out
