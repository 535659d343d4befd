"""Arrangements of a layer's parts around the residual stream.

`pre_norm` is GPT-2's: `x -> norm1 -> mixer -> +x -> norm2 -> feed-forward -> +x`, the residual
sums in float32 (graph_ir.cpp:732-756, the sequential branch; operand order x then the
branch's output, :754-756).  The mixer and the feed-forward add into the stream themselves so that
their last projection can do the sum in its epilogue.  A layer of this arrangement may have no
feed-forward (and then no second norm), and may add further things to the stream after its sublayers
(`LayerSpec.addons`).

`sandwich` norms every sublayer on both sides: `x -> x + after_mixer(mixer(norm1(x)))`, then
`x -> x + after_ffn(ffn(norm2(x)))`.  A sublayer's output cannot be added by its last projection
here (it is normed first), so the sublayer hands over its output as a weighted sum of float32
rows (`branches`) and the norm after it sums, norms and adds in one launch.  A layer of this
arrangement may have no feed-forward; it then has no norms around one either.

`shared_norm` has one norm that both sublayers read: `h = norm1(x)`, `x -> x + mixer(h) + ffn(h)`.
The mixer's last projection adds into the stream and the feed-forward's adds into that, both in
float32; a layer of this arrangement may have no feed-forward.

`post_norm` norms after the sum: `x -> norm1(alpha * x + mixer(x))`, then `x -> norm2(alpha * x + ffn(x))`, alpha a
constant (DeepNorm: Wang et al., "DeepNet: Scaling Transformers to 1,000 Layers").  The sublayers read the stream
itself, in the compute type; they hand over their outputs as branches and the norm's launch makes the sum, the norm, the
rows in the compute type and, where the layer's first addon is a sum over depth, that sum too.  A layer of this
arrangement may have no feed-forward and then has no second norm.
"""
from __future__ import annotations

from .base import Block, register_part


class PreNormBlock(Block):
    def __init__(self, norm1, mixer, norm2, ffn, **more_norms):
        if norm1 is None or more_norms or (ffn is None) != (norm2 is None):
            raise ValueError("block 'pre_norm' has a norm before the mixer and, with a feed-forward, one before that")
        super().__init__(norm1, mixer, norm2, ffn)


    def forward(self, ctx, x, app):
        announce = getattr(ctx.ops, "announce_weights", None)
        if announce is not None:    # a hint: this block's matrices in the order they are streamed, then what follows
            announce(self.mixer.stream_weights() + (self.ffn.stream_weights() if self.ffn is not None else [])
                     + list(getattr(ctx, "next_weights", ())))
        h = self.norm1.forward(ctx, x, ctx.dtype)
        x = self.mixer.forward(ctx, h, x, app)
        if self.ffn is not None:
            h = self.norm2.forward(ctx, x, ctx.dtype)
            ctx.rows_wanted = bool(self.addons)     # what follows reads the stream's rows in the compute type
            x = self.ffn.forward(ctx, h, x)
            ctx.rows_wanted = False
        return self.add_ons(ctx, x)


class SandwichBlock(Block):
    def __init__(self, norm1, mixer, norm2, ffn, after_mixer=None, after_ffn=None, **more_norms):
        if norm1 is None or after_mixer is None or more_norms:
            raise ValueError("block 'sandwich' has a norm before the mixer and one named 'after_mixer'")
        if (ffn is None) != (norm2 is None) or (ffn is None) != (after_ffn is None):
            raise ValueError("block 'sandwich' has a feed-forward with a norm before it and one named 'after_ffn', "
                             "or none of the three")
        extra = {"after_mixer": after_mixer} if ffn is None else {"after_mixer": after_mixer, "after_ffn": after_ffn}
        super().__init__(norm1, mixer, norm2, ffn, **extra)

    def forward(self, ctx, x, app):
        announce = getattr(ctx.ops, "announce_weights", None)
        if announce is not None:
            announce(self.mixer.stream_weights() + (self.ffn.stream_weights() if self.ffn is not None else [])
                     + list(getattr(ctx, "next_weights", ())))
        h = self.norm1.forward(ctx, x, ctx.dtype)
        x = self.more_norms["after_mixer"].add_normed(ctx, x, self.mixer.branches(ctx, h, app))
        if self.ffn is None:
            return x
        h = self.norm2.forward(ctx, x, ctx.dtype)
        return self.more_norms["after_ffn"].add_normed(ctx, x, self.ffn.branches(ctx, h))


class SharedNormBlock(Block):
    def __init__(self, norm1, mixer, norm2, ffn, **more_norms):
        if norm1 is None or norm2 is not None or more_norms:
            raise ValueError("block 'shared_norm' has exactly one norm, which the mixer and the feed-forward both read")
        super().__init__(norm1, mixer, None, ffn)

    def forward(self, ctx, x, app):
        announce = getattr(ctx.ops, "announce_weights", None)
        if announce is not None:
            announce(self.mixer.stream_weights() + (self.ffn.stream_weights() if self.ffn is not None else [])
                     + list(getattr(ctx, "next_weights", ())))
        h = self.norm1.forward(ctx, x, ctx.dtype)
        x = self.mixer.forward(ctx, h, x, app)
        return x if self.ffn is None else self.ffn.forward(ctx, h, x)


class PostNormBlock(Block):
    in_place = False

    def __init__(self, norm1, mixer, norm2, ffn, alpha: float = 1.0, **more_norms):
        if norm1 is None or more_norms or (ffn is None) != (norm2 is None):
            raise ValueError("block 'post_norm' has a norm after the mixer's sum and, with a feed-forward, one after that's")
        super().__init__(norm1, mixer, norm2, ffn)
        self.alpha = float(alpha)

    def forward(self, ctx, x, app):
        announce = getattr(ctx.ops, "announce_weights", None)
        if announce is not None:
            announce(self.mixer.stream_weights() + (self.ffn.stream_weights() if self.ffn is not None else [])
                     + list(getattr(ctx, "next_weights", ())))
        addons = list(self.addons)
        average = addons.pop(0) if addons and addons[0].reads_history else None
        branches = self.mixer.branches(ctx, ctx.rows_of(x), app)
        x = self.norm1.sum_normed(ctx, x, self.alpha, branches, average if self.ffn is None else None)
        if self.ffn is not None:
            x = self.norm2.sum_normed(ctx, x, self.alpha, self.ffn.row_branches(ctx, ctx.rows_of(x)), average)
        for part in addons:
            x = part.forward(ctx, x)
        return x


register_part("block", "post_norm", PostNormBlock)
register_part("block", "pre_norm", PreNormBlock)
register_part("block", "shared_norm", SharedNormBlock)
register_part("block", "sandwich", SandwichBlock)
