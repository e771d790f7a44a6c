"""Gated linear attention: a matrix state per head with a decay per key channel that depends on the
token, as a mixer over a running state instead of cached keys.

Per head, with q = Wq h * ``q_scale``, k = Wk h (``dim`` numbers), v = Wv h (``vdim``) and decays
through a low-rank pair of matrices,

    z = W2 (W1 h) + b          a = sigmoid(z)^(1 / tau)             (heads x dim; ``tau``)
    S_t = diag(a_t) S_(t-1) + k_t v_t^T          o_t = S_t^T q_t    (S_(-1) = 0)

each head's o is brought to unit root-mean-square, multiplied by a weight of ``vdim`` numbers that
the heads share and by silu(G h), and projected.  S is per-request STATE of the cache manager (a
slot per live request, zero at position 0), so a prompt may be cut anywhere and decoding is the
same recurrence with one token.  q, k, v, W1 and G are one product whose 32-bit result feeds the
recurrence unrounded; decays (which travel as a - 1), state and unit norm are 32-bit.  A step of
single tokens is one launch; steps with portions work out the decays and run the recurrence in
segments of 64 tokens side by side, with the finish inside the pass that has the outputs.  Sizes,
tau, the query's factor, eps and the constant on the result are parameters.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .interfaces import LayerCache, Mixer, StateSpec
from .latent_attention import FusedInput
from .linear import ResultProduct
from .registry import register_part


class GatedLinearAttention(Mixer):
    graph_safe = True
    can_overwrite = True
    takes_input_host = True

    def __init__(self, p: dict, store, runtime):
        w = p["weights"]
        self.width, self.heads = int(p["width"]), int(p["heads"])
        self.dim, self.vdim = int(p["dim"]), int(p["vdim"])
        self.eps, self.tau = float(p["eps"]), float(p.get("tau", 1.0))
        self.q_scale = float(p.get("q_scale", self.dim ** -0.5))
        self.out_scale = float(p.get("out_scale", 1.0))
        self.runtime = runtime
        if self.tau <= 0.0:
            raise ValueError("gated_linear_attention: tau must be positive")
        gpu = torch.cuda.is_available()
        self.scan_ok, self.finish_ok = ops.dscan_supports(self.dim, self.vdim) if gpu else (True, True)
        self.step_ok = gpu and ops.gla_step_supports(self.dim, self.vdim)
        if not self.scan_ok:
            raise ValueError(f"gated_linear_attention: heads of {self.dim} x {self.vdim} are beyond the "
                             f"scan's 512 numbers a key")

        def need(name, shape):
            t = store.get(w[name])
            if shape is not None and tuple(t.shape) != tuple(shape):
                raise ValueError(f"{w[name]}: expected {list(shape)}, found {list(t.shape)}")
            return t

        hk, hv = self.heads * self.dim, self.heads * self.vdim
        a1 = need("decay_down", None)
        if a1.dim() != 2 or a1.shape[1] != self.width:
            raise ValueError(f"{w['decay_down']}: expected [rank, {self.width}], found {list(a1.shape)}")
        self.rank = int(a1.shape[0])
        # the projections: one product of the mixer's own, or rows in the product of a mixer
        # beside it that reads the same input (``input_host``)
        self.host = p.get("input_host")
        self.input = None if self.host is not None else FusedInput(self.width, runtime, "gla_in")
        for name, rows in (("q", need("q", (hk, self.width))), ("k", need("k", (hk, self.width))),
                           ("v", need("v", (hv, self.width))), ("gate", need("gate", (hv, self.width))),
                           ("decay", a1)):
            if self.host is not None:
                self.host.fuse_input_rows("gla_" + name, rows)
            else:
                self.input.add(name, rows)
        f32 = lambda t: t.to(torch.float32).contiguous()
        # (the low rank outermost: a thread per channel reads neighbouring numbers)
        self.w2t = f32(need("decay_up", (hk, self.rank)).to(torch.float32).t())
        self.decay_bias = f32(need("decay_bias", (hk,)))
        self.norm = f32(need("norm", (self.vdim,)))
        self.out = ResultProduct(need("out", (self.width, hv)), runtime, "gla_gated")

    @property
    def accepts_lazy_norm(self) -> bool:
        return self.host is None

    def products(self):
        """(the fused first product or None, the product that ends the mixer)."""
        return self.input, self.out

    def state_specs(self):
        return [StateSpec("gla_state", (self.heads, self.vdim, self.dim), torch.float32)]

    def step_bytes(self, context: int) -> int:
        """State bytes a single token reads and writes back, whatever the context."""
        return 2 * 4 * self.heads * self.dim * self.vdim

    def forward(self, ctx, h, x, cache: LayerCache, accumulate: bool = True) -> None:
        t = x.shape[0]
        cap = ctx.token_capacity
        if self.host is not None:
            proj, host_cols = self.host.fused_product()
            c = {name: host_cols["gla_" + name][0] for name in ("q", "k", "v", "gate", "decay")}
        else:
            proj = self._proj = self.input.run(ctx, h)
            c = {name: at for name, (at, _n) in self.input.cols.items()}
        gated = self.out.buffer(ctx, t)
        state = cache.state["gla_state"]
        requests = ctx.layout.b_cap
        hk, hv = self.heads * self.dim, self.heads * self.vdim
        if ctx.max_q_len == 1 and self.step_ok:
            ops.gla_step(gated, proj, (c["q"], c["k"], c["v"], c["decay"], c["gate"]), self.w2t,
                         self.decay_bias, self.tau, self.q_scale, self.norm, state, ctx.q_start,
                         ctx.state_slot, ctx.positions, requests, self.heads, self.dim, self.vdim,
                         self.eps, self.out_scale, ctx.status)
        else:
            decay = ctx.scratch("gla_decay", (cap, hk), torch.float32)[:t]
            ops.gla_decay(decay, proj[:, c["decay"]:c["decay"] + self.rank], self.w2t, self.decay_bias,
                          self.tau)
            # (workspaces sized once, for the largest step the runtime takes)
            n = ops.dscan_max_segments(max(ctx.runtime.max_batched_tokens, ctx.layout.t_cap),
                                       max(ctx.runtime.max_requests, requests))
            big = (n, self.heads, self.vdim, self.dim)
            segments = (ctx.scratch("gla_seg_own", big, torch.float32),
                        ctx.scratch("gla_seg_start", big, torch.float32),
                        ctx.scratch("gla_seg_decay", (n, self.heads, self.dim), torch.float32))
            gate = proj[:, c["gate"]:c["gate"] + hv]
            raw = None if self.finish_ok else ctx.scratch("gla_raw", (cap, hv), torch.float32)[:t]
            ops.decayed_scan(raw, proj[:, c["q"]:c["q"] + hk], proj[:, c["k"]:c["k"] + hk],
                             proj[:, c["v"]:c["v"] + hv], decay, state, ctx.q_start, ctx.state_slot,
                             ctx.positions, requests, self.heads, self.dim, self.vdim, segments,
                             q_scale=self.q_scale, status=ctx.status,
                             finish=(gated, gate, self.norm, self.eps, self.out_scale)
                             if self.finish_ok else None)
            if not self.finish_ok:
                ops.gla_finish(gated, raw, gate, self.norm, ctx.seq_of_token, self.heads, self.vdim,
                               self.eps, self.out_scale)
        self.out.run(ctx, x, accumulate)


register_part("mixer", "gated_linear_attention", lambda p, store, rt: GatedLinearAttention(p, store, rt))
