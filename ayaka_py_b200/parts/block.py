"""Arrangements of a layer's parts."""

from __future__ import annotations

from .. import ops
from .base import Block, register_block


class PreNormBlock(Block):
    """x += mixer(norm1(x)); x += ffn(norm2(x))  (``models/gpt2.py:435-438``).
    The residual stream x is float32; the sums are made in the mixer's and the
    feed-forward's last epilogue."""

    KIND = "pre_norm"
    PARTS = ("norm1", "mixer", "norm2", "ffn")

    def forward(self, x, ctx, caches):
        x = self.mixer.forward(self.norm1.forward(x, ctx), x, ctx, caches.get("mixer"))
        return self.ffn.forward(self.norm2.forward(x, ctx), x, ctx)

    def lower(self, builder, x, caches):
        h = self.norm1.lower(builder, x)
        x = self.mixer.lower(builder, h, x, caches.get("mixer"))
        builder.release(h)
        h = self.norm2.lower(builder, x)
        x = self.ffn.lower(builder, h, x)
        builder.release(h)
        return x


class SandwichBlock(Block):
    """Norm before and after each sublayer, a short convolution over time in front of each:
    x += norm1b(mixer(conv1(norm1(x)))); x += norm2b(ffn(conv2(norm2(x)))).  The closing norms carry
    the residual multiplier and add to the stream themselves (``RMSNorm.add_normed``); the norm
    in front and the convolution are one kernel (``TimeConv.forward``)."""

    KIND = "sandwich"
    PARTS = ("norm1", "conv1", "mixer", "norm1b", "norm2", "conv2", "ffn", "norm2b")

    def forward(self, x, ctx, caches):
        h = self.conv1.forward(x, self.norm1, ctx, caches["conv1"])
        x = self.norm1b.add_normed(x, self.mixer.forward(h, None, ctx, caches.get("mixer")))
        if "ffn" in self.parts:
            h = self.conv2.forward(x, self.norm2, ctx, caches["conv2"])
            x = self.norm2b.add_normed(x, self.ffn.forward(h, None, ctx))
        return x


class SandwichMixerBlock(SandwichBlock):
    """The same without a feed-forward."""

    KIND = "sandwich_mixer_only"
    PARTS = ("norm1", "conv1", "mixer", "norm1b")


register_block(PreNormBlock.KIND, PreNormBlock)
register_block(SandwichBlock.KIND, SandwichBlock)
register_block(SandwichMixerBlock.KIND, SandwichMixerBlock)


class PostNormBlock(Block):
    """The sublayers read the residual stream itself and only their outputs are normed:
    x += norm1(mixer(shift(x))); x += norm2(ffn(x)).  ``shift`` blends every channel of the
    mixer's input with the previous token's (``TokenShift``); it also brings the stream into the
    compute dtype, which a plain conversion does for the feed-forward.  The closing norms carry
    the residual multiplier and add to the stream themselves (``RMSNorm.add_normed``)."""

    KIND = "post_norm"
    PARTS = ("shift", "mixer", "norm1", "ffn", "norm2")

    def forward(self, x, ctx, caches):
        h = self.shift.forward(x, ctx, caches["shift"])
        x = self.norm1.add_normed(x, self.mixer.forward(h, None, ctx, caches.get("mixer")))
        if "ffn" in self.parts:
            x = self.norm2.add_normed(x, self.ffn.forward(self.shift.convert(x), None, ctx))
        return x


class PostNormMixerBlock(PostNormBlock):
    """The same without a feed-forward."""

    KIND = "post_norm_mixer_only"
    PARTS = ("shift", "mixer", "norm1")


register_block(PostNormBlock.KIND, PostNormBlock)
register_block(PostNormMixerBlock.KIND, PostNormMixerBlock)


class DoubleNormBlock(Block):
    """Norm before and after each sublayer, nothing else between:
    x += norm1b(mixer(norm1(x))); x += norm2b(ffn(norm2(x))).  The closing norms add to the stream
    themselves (``RMSNorm.add_normed``); the mixer's closing norm and the feed-forward's opening norm are
    one kernel (``RMSNorm.add_normed_then``)."""

    KIND = "double_norm"
    PARTS = ("norm1", "mixer", "norm1b", "norm2", "ffn", "norm2b")

    def forward(self, x, ctx, caches):
        y = self.mixer.forward(self.norm1.forward(x, ctx), None, ctx, caches.get("mixer"))
        if "ffn" not in self.parts:
            return self.norm1b.add_normed(x, y)
        h = self.norm1b.add_normed_then(x, y, self.norm2)
        return self.norm2b.add_normed(x, self.ffn.forward(h, None, ctx))


class DoubleNormMixerBlock(DoubleNormBlock):
    """The same without a feed-forward."""

    KIND = "double_norm_mixer_only"
    PARTS = ("norm1", "mixer", "norm1b")


register_block(DoubleNormBlock.KIND, DoubleNormBlock)
register_block(DoubleNormMixerBlock.KIND, DoubleNormMixerBlock)


class GatedPreNormBlock(Block):
    """A norm in front of each sublayer, a constant and a gate per channel behind it (``ResidualGate``), and a token's
    row of a side table at the layer's end (``TokenSide``):
    x += s1 g1(h) mixer(h) with h = norm1(x); x += s2 g2(h) ffn(h) with h = norm2(x); x += side(x, token).
    The feed-forward (with its norm and gate) and the side input may be absent.  The gates' products ride in the
    sublayers' first products; every update of the stream is one kernel that also makes what the next product reads
    (``ops.stream_update``), the next layer's opening norm included."""

    KIND = "gated_pre_norm"
    PARTS = ("norm1", "mixer", "gate1")
    OPTIONAL = ("norm2", "ffn", "gate2", "side")

    def __init__(self, parts):
        super().__init__(parts)
        together = [name in parts for name in ("norm2", "ffn", "gate2")]
        if any(together) and not all(together):
            raise ValueError(f"arrangement {self.KIND!r}: norm2, ffn and gate2 come together or not at all")

    def bound(self):
        self.gate1.ride(self.mixer)
        if "ffn" in self.parts:
            self.gate2.ride(self.ffn)

    def opening_norm(self):
        return self.norm1

    @staticmethod
    def _update(x, y, norm, ctx, **how):
        """The stream takes up y; returns ``norm`` of it (None: nothing), from the same kernel where that can be."""
        post = norm.as_following() if norm is not None else None
        h = ops.stream_update(x, y, **how, **(post or {}))
        return norm.forward(x, ctx) if norm is not None and post is None else h

    def forward(self, x, ctx, caches):
        h = ctx.carry.pop("opened", None)
        if h is None:
            h = self.norm1.forward(x, ctx)
        y, gate = self.mixer.forward(h, None, ctx, caches.get("mixer")), self.gate1
        gates = gate.gates(self.mixer, h, ctx)
        if "ffn" in self.parts:
            h = self._update(x, y, self.norm2, ctx, scale=gate.scale, gate=gates)
            y, gate = self.ffn.forward_rows(h, ctx), self.gate2
            gates = gate.gates(self.ffn, h, ctx)
        if "side" in self.parts:
            copies = {"post": "copy", "out_dtype": self.side.dtype} if self.side.reads_copy(x.shape[0]) else {}
            copy = ops.stream_update(x, y, gate.scale, gate=gates, **copies)
            opened = self._update(x, self.side.forward(x, copy, ctx), ctx.following, ctx, scale=self.side.norm, eps=self.side.eps)
        else:
            opened = self._update(x, y, ctx.following, ctx, scale=gate.scale, gate=gates)
        if opened is not None:
            ctx.carry["opened"] = opened
        return x


register_block(GatedPreNormBlock.KIND, GatedPreNormBlock)


class NormedSumBlock(Block):
    """The sublayers read the stream itself (``StreamCopy``) and a norm closes every sum, the stream with a factor of its
    own in it: x = norm1(a x + mixer(x)); x = norm2(a x + ffn(x)).  The feed-forward (with its norm) may be absent.
    Every sum, its norm and the copy that the next sublayer reads are one kernel (``RMSNorm.sum_normed``), which also
    adds up a routed feed-forward's rows."""

    KIND = "normed_sum"
    PARTS = ("copy", "mixer", "norm1")
    OPTIONAL = ("ffn", "norm2")

    def __init__(self, parts):
        super().__init__(parts)
        if ("ffn" in parts) != ("norm2" in parts):
            raise ValueError(f"arrangement {self.KIND!r}: ffn and norm2 come together or not at all")

    def opening_norm(self):
        return self.copy

    def forward(self, x, ctx, caches):
        h = ctx.carry.pop("opened", None)
        if h is None:
            h = self.copy.forward(x, ctx)
        y, norm = self.mixer.forward(h, None, ctx, caches.get("mixer")), self.norm1
        if "ffn" in self.parts:
            h = norm.sum_normed(x, y, self.copy, ctx)
            y, norm = self.ffn.forward_rows(h, ctx), self.norm2
        opened = norm.sum_normed(x, y, ctx.following, ctx)
        if opened is not None:
            ctx.carry["opened"] = opened
        return x


register_block(NormedSumBlock.KIND, NormedSumBlock)
