"""Ways to join the stream with its own beginning between layers.  ``linear_join``:
x <- W [x; x0] with x0 the embedding's output and W [width, 2 width], a matrix product with a
32-bit result.  Its input is one buffer per step, [x | x0] in the activation type: the
embedding writes both halves, and a block whose successor is a join leaves its stream there
(``ctx.wanted_after``), so that nothing is copied between."""
from __future__ import annotations

import torch

from .interfaces import StreamJoin
from .linear import padded_linear
from .registry import register_part


class LinearJoin(StreamJoin):
    graph_safe = True

    def __init__(self, weight: torch.Tensor, width: int, runtime):
        if tuple(weight.shape) != (width, 2 * width):
            raise ValueError(f"linear_join: the matrix is {list(weight.shape)}, expected "
                             f"[{width}, {2 * width}]")
        self.linear = padded_linear(weight, runtime)
        self.width, self.runtime = width, runtime

    def buffer(self, ctx, rows: int) -> torch.Tensor:
        return ctx.scratch_zero("stream_join_in", (ctx.token_capacity, self.linear.n_in),
                                self.runtime.dtype)[:rows]

    def forward(self, ctx, pair: torch.Tensor, x: torch.Tensor) -> None:
        self.linear.forward(ctx, pair, x)


register_part("stream_join", "linear_join",
              lambda p, store, rt: LinearJoin(store.get(p["weights"]), p["width"], rt))
