"""Arrangements of parts in a block.  ``pre_norm``:
x += mixer(norm_1(x)); x += feed_forward(norm_2(x))  (``dev/examples/gpt2.clj:149-166``).
The block knows its parts only through their interfaces."""
from __future__ import annotations

from typing import Dict

import torch

from ..csrc import ops
from ..settings import SETTINGS
from .interfaces import Block, FeedForward, LayerCache, Mixer, Norm
from .linear import LazyNorm, Linear
from .registry import register_part


class PreNormBlock(Block):
    graph_safe = True
    def __init__(self, mixer: Mixer, feed_forward: FeedForward, norms: Dict[str, Norm],
                 width: int, runtime):
        # (a layer without a feed-forward has the mixer's norm alone)
        self.has_ff = not getattr(feed_forward, "is_none", False)
        wanted = {"mixer", "feed_forward"} if self.has_ff else {"mixer"}
        if set(norms) != wanted:
            raise ValueError(f"pre_norm wants the norms {sorted(wanted)}, got {sorted(norms)}")
        self.mixer, self.feed_forward = mixer, feed_forward
        self.norms = dict(norms)
        self.mixer_norm, self.feed_forward_norm = norms["mixer"], norms.get("feed_forward")
        self.width, self.runtime = width, runtime

    def forward(self, ctx, x, cache: LayerCache) -> None:
        t = x.shape[0]
        h = ctx.scratch("block_normed", (ctx.token_capacity, self.width), self.runtime.dtype)[:t]
        self.mixer.forward(ctx, self._normed(ctx, self.mixer, self.mixer_norm, x, h), x, cache)
        if not self.has_ff:
            return
        self.feed_forward.forward(
            ctx, self._normed(ctx, self.feed_forward, self.feed_forward_norm, x, h), x)

    @staticmethod
    def _normed(ctx, consumer, norm, x, out):
        """The consumer's input: a norm that has run, or, for consumers that say they take
        one (``accepts_lazy_norm``), a :class:`LazyNorm` they may fuse into their first
        matrix product."""
        lazy = LazyNorm(ctx, norm, x, out)
        return lazy if getattr(consumer, "accepts_lazy_norm", False) else lazy.tensor()


class PostNormGatedBlock(Block):
    """x <- norm_1(alpha x + g_1(x) * mixer(x)); x <- norm_2(alpha x + g_2(x) * feed_forward(x)):
    the branches read the stream itself, the norm comes after the sum, and a branch's result may
    be gated element by element by g(x) = sigmoid(W x + b) (``params["gates"]``: branch name ->
    tensor name of W, with ``.b``).  A layer without a feed-forward has the first half only
    (and, if its file still holds a second norm, ``params["norm_alone"]``, that norm of the
    scaled stream).

    The gate's matrix rides along in the branch's first matrix product where the part offers
    that (``fuse_input_rows``); sum, gate and norm are one kernel, which also leaves the
    stream's copy in the activation type for the next branch's product."""
    graph_safe = True

    def __init__(self, mixer: Mixer, feed_forward: FeedForward, norms: Dict[str, Norm],
                 width: int, runtime, params=None, store=None):
        params = params or {}
        self.mixer, self.feed_forward = mixer, feed_forward
        self.norms = dict(norms)
        self.width, self.runtime = width, runtime
        self.alpha = float(params.get("alpha", 1.0))
        self.has_ff = not getattr(feed_forward, "is_none", False)
        wanted = {"mixer"} | ({"feed_forward"} if self.has_ff else set())
        if set(norms) != wanted:
            raise ValueError(f"post_norm_gated wants the norms {sorted(wanted)}, got {sorted(norms)}")
        for part in (mixer, feed_forward):
            if not getattr(part, "can_overwrite", False):
                raise ValueError(f"post_norm_gated: {type(part).__name__} cannot hand over its "
                                 f"result apart from the stream")
        for norm in norms.values():
            if not hasattr(norm, "joined"):
                raise ValueError("post_norm_gated needs norms that can join a branch to the stream")
        # a layer without a feed-forward whose file still holds the second norm: x <- norm(alpha x)
        self.norm_alone = None
        alone = params.get("norm_alone")
        if not self.has_ff and alone and store is not None and alone["gain"] in store:
            from .norms import RMSNorm
            self.norm_alone = RMSNorm(store.get(alone["gain"]), None, alone["eps"], width)
            self.norms["alone"] = self.norm_alone
        self.gates = {}
        for name, tensor in (params.get("gates") or {}).items():
            part = {"mixer": mixer, "feed_forward": feed_forward}[name]
            w, b = store.get(tensor), store.get(tensor + ".b")
            if tuple(w.shape) != (width, width) or b.numel() != width:
                raise ValueError(f"{tensor}: a gate of the stream is [{width}, {width}] with a bias")
            bias = b.to(torch.float32).contiguous()
            if hasattr(part, "fuse_input_rows"):
                self.gates[name] = (part.fuse_input_rows("branch_gate", w), None, bias)
            else:
                self.gates[name] = (None, Linear(w, None, runtime), bias)

    def forward(self, ctx, x, cache: LayerCache) -> None:
        t = x.shape[0]
        cap = ctx.token_capacity
        y = ctx.scratch("branch_result", (cap, self.width), torch.float32)[:t]
        serving = self.runtime.dtype != torch.float32
        copy = ctx.scratch("stream_copy", (cap, self.width), self.runtime.dtype)[:t] if serving else None
        # the stream in the products' type: the norm before left it, unless this is the model's
        # first branch or another kind of block has changed the stream since
        writer = getattr(ctx, "stream_copy_by", None)
        current = writer is not None and writer is getattr(ctx, "last_block", None)
        for name, part in (("mixer", self.mixer), ("feed_forward", self.feed_forward)):
            if name == "feed_forward" and not self.has_ff:
                break
            h = x
            if serving:
                if not current:
                    ops.bias_act(copy, x, None, None, None)
                h = copy
            if name == "mixer":
                part.forward(ctx, h, y, cache, accumulate=False)
            else:
                part.forward(ctx, h, y, accumulate=False)
            gate = bias = None
            if name in self.gates:
                fused, own, bias = self.gates[name]
                if fused is not None:
                    gate = part.fused_rows(fused)
                else:
                    gate = ctx.scratch("branch_gate", (cap, self.width), torch.float32)[:t]
                    own.forward(ctx, h, gate)
            self.norms[name].joined(ctx, x, y, self.alpha, gate=gate, gate_bias=bias, copy=copy)
            current = True
        if self.norm_alone is not None:
            self.norm_alone.joined(ctx, x, None, self.alpha, copy=copy)
        ctx.stream_copy_by = self


class ParallelBlock(Block):
    """x <- x + (mixer(norm_1(x)) + feed_forward(norm_2(x))): both branches read the stream as
    it was before the layer, each through a norm of its own, and their results join it in
    32-bit.  The mixer's norm runs first; the feed-forward then reads the untouched stream
    (its norm may ride in its first matrix product, see :class:`LazyNorm`) and adds its
    result, and the mixer, which works from its normed copy, adds its own after that.  A
    layer without a feed-forward has the mixer's norm alone.

    With ONE norm (``norms`` = {"shared"}) both branches read its result: x <- x + (mixer(h) +
    feed_forward(h)), h = norm(x).  Branches that offer their products (``products``: the fused first
    product and the product that ends them) then share both: one product reads h for all of the
    layer's projections, and one brings all of its results to the stream; the norm may ride in the
    first (the stream stays as it was until the last)."""
    graph_safe = True

    def __init__(self, mixer: Mixer, feed_forward: FeedForward, norms: Dict[str, Norm],
                 width: int, runtime):
        self.has_ff = not getattr(feed_forward, "is_none", False)
        self.shared = set(norms) == {"shared"}
        wanted = {"mixer", "feed_forward"} if self.has_ff else {"mixer"}
        if not self.shared and set(norms) != wanted:
            raise ValueError(f"parallel wants the norms {sorted(wanted)} or ['shared'], got {sorted(norms)}")
        self.mixer, self.feed_forward = mixer, feed_forward
        self.norms = dict(norms)
        self.width, self.runtime = width, runtime
        self.result = None                  # the branches' common last product, if they have one
        if self.shared and self.has_ff:
            mine = getattr(mixer, "products", lambda: None)()
            theirs = getattr(feed_forward, "products", lambda: None)()
            if mine is not None and theirs is not None:
                mine[0].absorb(theirs[0])
                mine[1].absorb(theirs[1])
                self.result = mine[1]
                self.result.closer = self

    def _forward_shared(self, ctx, x, cache: LayerCache) -> None:
        h = ctx.scratch("block_normed", (ctx.token_capacity, self.width), self.runtime.dtype)[:x.shape[0]]
        norm = self.norms["shared"]
        if self.result is not None or not self.has_ff:
            h_in = PreNormBlock._normed(ctx, self.mixer, norm, x, h)
            if self.has_ff and SETTINGS.side_streams and getattr(self.feed_forward, "worth_a_branch", False):
                # the feed-forward's activations beside the mixer: both start from the first product
                self.mixer.products()[0].run_ahead(ctx, h_in)
                self.result.buffer(ctx, x.shape[0])        # (there before the branches part)
                side = ctx.side(1)
                with side, ops.plain_launch():
                    self.feed_forward.forward(ctx, h_in, x)
                self.mixer.forward(ctx, h_in, x, cache)
                side.join()
                with ops.plain_launch():
                    self.result.close(ctx, x)
                return
            self.mixer.forward(ctx, h_in, x, cache)
            if self.has_ff:
                self.feed_forward.forward(ctx, h_in, x)
                self.result.close(ctx, x)
            return
        norm.forward(ctx, x, h)
        self.mixer.forward(ctx, h, x, cache)
        self.feed_forward.forward(ctx, h, x)

    def forward(self, ctx, x, cache: LayerCache) -> None:
        if self.shared:
            self._forward_shared(ctx, x, cache)
            return
        t = x.shape[0]
        cap = ctx.token_capacity
        h1 = ctx.scratch("block_normed", (cap, self.width), self.runtime.dtype)[:t]
        self.norms["mixer"].forward(ctx, x, h1)
        if self.has_ff:
            h2 = ctx.scratch("block_normed_2", (cap, self.width), self.runtime.dtype)[:t]
            self.feed_forward.forward(
                ctx, PreNormBlock._normed(ctx, self.feed_forward, self.norms["feed_forward"], x, h2), x)
        self.mixer.forward(ctx, h1, x, cache)


class BranchNormBlock(Block):
    """x <- x + norm_1(mixer(x)); x <- x + norm_2(feed_forward(x)): the branches read the stream
    itself and each branch's RESULT is normed before it joins the stream.  A layer without a
    feed-forward has the first half only.  Norm and sum are one kernel, which also leaves the
    stream's copy in the activation type for the next branch's product."""
    graph_safe = True

    def __init__(self, mixer: Mixer, feed_forward: FeedForward, norms: Dict[str, Norm],
                 width: int, runtime):
        self.mixer, self.feed_forward = mixer, feed_forward
        self.norms = dict(norms)
        self.width, self.runtime = width, runtime
        self.has_ff = not getattr(feed_forward, "is_none", False)
        wanted = {"mixer"} | ({"feed_forward"} if self.has_ff else set())
        if set(norms) != wanted:
            raise ValueError(f"branch_norm wants the norms {sorted(wanted)}, got {sorted(norms)}")
        for part in (mixer, feed_forward):
            if not getattr(part, "can_overwrite", False):
                raise ValueError(f"branch_norm: {type(part).__name__} cannot hand over its result "
                                 f"apart from the stream")
        for norm in norms.values():
            if not hasattr(norm, "added"):
                raise ValueError("branch_norm needs norms that can add a normed branch to the stream")

    def forward(self, ctx, x, cache: LayerCache) -> None:
        t = x.shape[0]
        cap = ctx.token_capacity
        y = ctx.scratch("branch_result", (cap, self.width), torch.float32)[:t]
        serving = self.runtime.dtype != torch.float32
        copy = ctx.scratch("stream_copy", (cap, self.width), self.runtime.dtype)[:t] if serving else None
        # the stream in the products' type: the norm before left it, unless this is the model's
        # first branch or another kind of block has changed the stream since
        writer = getattr(ctx, "stream_copy_by", None)
        current = writer is not None and writer is getattr(ctx, "last_block", None)
        for name, part in (("mixer", self.mixer), ("feed_forward", self.feed_forward)):
            if name == "feed_forward" and not self.has_ff:
                break
            h = x
            if serving:
                if not current:
                    ops.bias_act(copy, x, None, None, None)
                h = copy
            if name == "mixer":
                part.forward(ctx, h, y, cache, accumulate=False)
            else:
                part.forward(ctx, h, y, accumulate=False)
            self.norms[name].added(ctx, x, y, copy=copy)
            current = True
        ctx.stream_copy_by = self


class SandwichBlock(Block):
    """x <- x + m * norm_1b(mixer(norm_1(x))); x <- x + m * norm_2b(feed_forward(norm_2(x))): a norm
    before and a norm after each branch, and a constant m (``params["residual_mult"]``) on what
    joins the stream.  A layer without a feed-forward has the first half only.

    A branch's second norm, the sum and the NEXT branch's first norm are one kernel, also across
    layers: ``ctx.wanted_after`` says what reads the stream next (a norm, or a buffer that takes
    a copy of it), and what this block leaves for it is ``ctx.stream_left``."""
    graph_safe = True

    def __init__(self, mixer: Mixer, feed_forward: FeedForward, norms: Dict[str, Norm],
                 width: int, runtime, params=None, store=None):
        self.mixer, self.feed_forward = mixer, feed_forward
        self.norms = dict(norms)
        self.width, self.runtime = width, runtime
        self.mult = float((params or {}).get("residual_mult", 1.0))
        self.has_ff = not getattr(feed_forward, "is_none", False)
        wanted = {"mixer", "mixer_after"} | ({"feed_forward", "feed_forward_after"} if self.has_ff else set())
        if set(norms) != wanted:
            raise ValueError(f"sandwich wants the norms {sorted(wanted)}, got {sorted(norms)}")
        for part in (mixer, feed_forward):
            if not getattr(part, "can_overwrite", False):
                raise ValueError(f"sandwich: {type(part).__name__} cannot hand over its result apart "
                                 f"from the stream")
        for name in ("mixer_after", "feed_forward_after"):
            if name in norms and getattr(norms[name], "pair", lambda: None)() is None:
                raise ValueError("sandwich needs norms with a weight per coordinate after the branches")
        #: the norm this block reads the stream through first
        self.entry_norm = norms["mixer"]

    def forward(self, ctx, x, cache: LayerCache) -> None:
        t = x.shape[0]
        cap = ctx.token_capacity
        y = ctx.scratch("branch_result", (cap, self.width), torch.float32)[:t]
        h = ctx.scratch("block_normed", (cap, self.width), self.runtime.dtype)[:t]
        arrived = getattr(ctx, "arrived", None)
        ready = arrived is not None and arrived[0] is self.entry_norm
        h_in = arrived[1] if ready else PreNormBlock._normed(ctx, self.mixer, self.entry_norm, x, h)
        self.mixer.forward(ctx, h_in, y, cache, accumulate=False)
        after = getattr(ctx, "wanted_after", None)
        if self.has_ff:
            norm = self.norms["feed_forward"]
            ready = self._join(x, y, "mixer_after", norm, h)
            h_in = h if ready else PreNormBlock._normed(ctx, self.feed_forward, norm, x, h)
            self.feed_forward.forward(ctx, h_in, y, accumulate=False)
        if self._join(x, y, "feed_forward_after" if self.has_ff else "mixer_after", after, h):
            ctx.stream_left = (after, h)

    def _join(self, x, y, name: str, reader, h) -> bool:
        """x <- x + m * norm(y), and what ``reader`` wants of the new x: a norm's result in ``h``,
        or a copy in the buffer it is.  True if that has been done."""
        weight, bias, eps, centred = self.norms[name].pair()
        if isinstance(reader, torch.Tensor):
            ops.norm_pair(x, y, self.mult, weight, bias, eps, centred, out=reader)
            return True
        following = getattr(reader, "pair", lambda: None)()
        ops.norm_pair(x, y, self.mult, weight, bias, eps, centred,
                      out=None if following is None else h, next_norm=following)
        return following is not None


register_part("arrangement", "pre_norm", PreNormBlock)
register_part("arrangement", "sandwich", SandwichBlock)
register_part("arrangement", "branch_norm", BranchNormBlock)
register_part("arrangement", "post_norm_gated", PostNormGatedBlock)
register_part("arrangement", "parallel", ParallelBlock)
