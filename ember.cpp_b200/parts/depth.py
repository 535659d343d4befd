"""A weighted sum over depth: what goes on after a layer is a sum of that layer's result and of everything in front of it.

With X_0 the stream that the embedding left and X_(i+1) the result of layer i, the stream after layer i is
sum over j = 0 .. i+1 of w_j X_j, the weights being one stored vector a layer (Pagliardini et al., "DenseFormer: Enhancing
Information Flow in Transformers via Depth Weighted Averaging").  X_(i+1) is the layer's result before the sum.

The results are kept for the step in `ctx.history` (the model puts X_0 there).  An arrangement whose last launch norms
the stream can take the sum into that launch: it asks `fold(ctx)` for the tensors in front and the weights, and hands the
result to `keep(ctx, y)`; any other arrangement runs `forward`.
"""
from __future__ import annotations

from .base import StreamAddon, WeightSpec, register_part


class DepthAverage(StreamAddon):
    reads_history = True

    def __init__(self, prefix: str, layers: int, weights: str = "dwa", init_std: float = 0.1):
        """layers: how many results stand in front of this layer's own (the embedding's included)."""
        super().__init__(prefix)
        self.layers, self.weights_name, self.init_std = int(layers), prefix + weights, init_std
        if self.layers < 1:
            raise ValueError(f"depth average {prefix!r}: {self.layers} results in front")
        self.weights = None

    def weight_specs(self):
        # random-weights mode: every term about alike, so that the stream keeps its size
        return [WeightSpec(self.weights_name, (self.layers + 1,), mean=1.0 / (self.layers + 1), std=self.init_std)]

    def load(self, get, runtime):
        self.weights = runtime.vector(get(self.weights_name))

    def fold(self, ctx):
        if len(ctx.history) != self.layers:
            raise ValueError(f"depth average {self.prefix!r}: {len(ctx.history)} results in front, weights for {self.layers}")
        return list(ctx.history), self.weights

    def keep(self, ctx, y) -> None:
        ctx.history.append(y)

    def forward(self, ctx, x):
        history, weights = self.fold(ctx)
        self.keep(ctx, x)
        stream, rows = ctx.ops.depth_average(history + [x], weights, ctx.dtype)
        ctx.note_rows(stream, rows)
        return stream


register_part("addon", "depth_average", DepthAverage)
