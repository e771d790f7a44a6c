"""Output head.  ``tied_head``: logits[r, v] = sum_d h[r, d] * table[v, d] with the token
table as the matrix and no bias (``dev/examples/gpt2.clj:108-122``); logits are float32."""
from __future__ import annotations

import torch

from ..csrc import ops
from .interfaces import Head
from .linear import Linear
from .registry import register_part


class TiedHead(Head):
    graph_safe = True
    accepts_lazy_norm = True        # ``h`` may be a LazyNorm: few rows are normed inside the product
    def __init__(self, table: torch.Tensor, vocab: int, width: int, runtime):
        if tuple(table.shape) != (vocab, width):
            raise ValueError(f"tied_head: table is {list(table.shape)}, expected [{vocab}, {width}]")
        self.linear = Linear(table, None, runtime)      # [vocab, width] is already [out, in]
        self.vocab = vocab

    def forward(self, ctx, h, logits) -> None:
        self.linear.forward(ctx, h, logits)


class LinearHead(TiedHead):
    """A head with a matrix of its own, [vocab, width], no bias.  ``softcap`` > 0: the logits are
    softcap * tanh(logits / softcap)."""

    def __init__(self, table: torch.Tensor, vocab: int, width: int, runtime, softcap: float = 0.0):
        super().__init__(table, vocab, width, runtime)
        self.softcap = float(softcap or 0.0)
        if self.softcap < 0.0:
            raise ValueError(f"linear_head: a cap of {self.softcap} on the logits")

    def forward(self, ctx, h, logits) -> None:
        super().forward(ctx, h, logits)
        if self.softcap > 0.0:
            ops.tanh_cap(logits, self.softcap)


register_part("head", "linear_head",
              lambda p, store, rt: LinearHead(store.get(p["weights"], rt.dtype), p["vocab"],
                                              p["width"], rt, p.get("softcap", 0.0)))
register_part("head", "tied_head",
              lambda p, store, rt: TiedHead(store.get(p["weights"] + ".weight", rt.dtype),
                                            p["vocab"], p["width"], rt))
