"""Mamba-2's state-space mixer (Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient
Algorithms Through Structured State Space Duality"), over a running state instead of cached keys.

One matrix gives a token's [z | x B C | dt]: z and x are ``heads`` * ``vdim`` wide, B and C ``groups``
rows of ``state`` numbers (head h uses group h / (heads / groups)), dt one number a head.

    xBC = silu(conv(x B C) + b)       a causal convolution per channel, ``taps`` long, the last tap on
                                      the current token, zeros before the sequence's start
    dt  = softplus(dt + dt_bias)      a = exp(-exp(A_log) dt)
    S_t = a_t S_(t-1) + dt_t B_t x_t^T           y_t = S_t^T C_t + D x_t          (S_(-1) = 0)

y (heads side by side) is multiplied by silu(z), RMS-normed in ``norm_parts`` equal parts, multiplied
by a weight and projected.  S and the convolution's last inputs are per-request STATE of the cache
manager (a slot per live request, zero at position 0; the input of position p lies in row p mod
``taps``), so a prompt may be cut anywhere.

A step of single tokens is one launch.  Steps with portions: convolution, step sizes and decays; the
recurrence in segments of 64 tokens side by side; the norm.  In bfloat16 the segments' products run
on tensor cores (convolved x, B and C are bfloat16 operands; scores, decays, step sizes and states
are 32-bit and enter products as pairs of bfloat16 numbers); in 32-bit, and for sizes those kernels do
not take, the recurrence of :func:`~pretrained_rstr_b200.csrc.ops.decayed_scan` runs instead.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .interfaces import LayerCache, Mixer, StateSpec
from .latent_attention import FusedInput
from .linear import ResultProduct
from .registry import register_part


class StateSpace(Mixer):
    graph_safe = True
    can_overwrite = True
    accepts_lazy_norm = True      # the first matrix product may compute the norm itself

    def __init__(self, p: dict, store, runtime):
        w = p["weights"]
        self.width, self.heads, self.vdim = int(p["width"]), int(p["heads"]), int(p["vdim"])
        self.state_dim, self.groups, self.taps = int(p["state"]), int(p["groups"]), int(p["taps"])
        self.parts, self.eps = int(p.get("norm_parts", 1)), float(p["eps"])
        self.out_scale = float(p.get("out_scale", 1.0))
        self.runtime = runtime
        inner, bc = self.heads * self.vdim, 2 * self.groups * self.state_dim
        self.inner, self.channels = inner, inner + bc
        if self.heads % self.groups or inner % self.parts:
            raise ValueError(f"state_space: {self.heads} heads of {self.vdim} do not split into "
                             f"{self.groups} groups and {self.parts} parts of the norm")
        gpu = torch.cuda.is_available()
        if self.taps < 1 or (gpu and self.taps > ops.ssm_max_taps()):
            raise ValueError(f"state_space: a convolution of {self.taps} taps is not built")
        if gpu and not ops.dscan_supports(self.state_dim, self.vdim)[0]:
            raise ValueError(f"state_space: heads of {self.state_dim} x {self.vdim} are beyond the "
                             f"scan's 512 numbers a key")

        def need(name, shape):
            t = store.get(w[name])
            if tuple(t.shape) != tuple(shape):
                raise ValueError(f"{w[name]}: expected {list(shape)}, found {list(t.shape)}")
            return t

        f32 = lambda t: t.to(torch.float32).contiguous()
        rows = need("in", (inner + self.channels + self.heads, self.width))
        self.input = FusedInput(self.width, runtime, "ssm_in")
        self.input.add("z", rows[:inner])
        self.input.add("xbc", rows[inner:inner + self.channels])
        self.input.add("dt", rows[inner + self.channels:])
        # (the tap outermost: a thread per channel reads neighbouring numbers)
        self.conv_w = f32(need("conv", (self.channels, self.taps)).to(torch.float32).t())
        self.conv_b = f32(need("conv_bias", (self.channels,)))
        self.dt_bias = f32(need("dt_bias", (self.heads,)))
        self.neg_a = (-torch.exp(f32(need("A_log", (self.heads,))))).contiguous()
        self.direct = f32(need("D", (self.heads,)))
        self.norm = f32(need("norm", (inner,)))
        self.out = ResultProduct(need("out", (self.width, inner)), runtime, "ssm_gated")
        self.chunks_ok = gpu and runtime.dtype == torch.bfloat16 and \
            ops.ssm_chunk_supports(self.vdim, self.state_dim)

    def products(self):
        """(the fused first product, the product that ends the mixer)."""
        return self.input, self.out

    def fuse_input_rows(self, name: str, weight) -> str:
        return self.input.add(name, weight)

    def fused_rows(self, name: str):
        return self.input.view(self._proj, name)

    def fused_product(self):
        """(the fused product's 32-bit result of this step, first column by segment name): for a
        mixer beside this one whose projections ride in the product."""
        return self.input.result, self.input.cols

    def state_specs(self):
        specs = [StateSpec("ssm_state", (self.heads, self.vdim, self.state_dim), torch.float32)]
        if self.taps > 1:
            specs.append(StateSpec("ssm_inputs", (self.taps, self.channels), torch.float32))
        return specs

    def step_bytes(self, context: int) -> int:
        """State bytes a single token reads and writes back, whatever the context."""
        return 2 * 4 * (self.inner * self.state_dim + (self.taps - 1) * self.channels)

    def forward(self, ctx, h, x, cache: LayerCache, accumulate: bool = True) -> None:
        t = x.shape[0]
        cap = ctx.token_capacity
        proj = self._proj = self.input.run(ctx, h)
        cols = tuple(self.input.cols[name][0] for name in ("z", "xbc", "dt"))
        requests = ctx.layout.b_cap
        state = cache.state["ssm_state"]
        raw = ctx.scratch("ssm_raw", (cap, self.inner), torch.float32)[:t]
        kernels = ops.StateSpace(
            proj, cols, self.conv_w, self.conv_b, self.dt_bias, self.neg_a, self.direct, self.norm,
            cache.state.get("ssm_inputs"), state, ctx.seq_of_token, ctx.q_start, ctx.state_slot,
            ctx.positions, requests, self.heads, self.vdim, self.state_dim, self.groups, self.parts,
            self.eps, self.out_scale, raw, self.out.buffer(ctx, t), ctx.status)
        if ctx.max_q_len == 1:
            kernels.step(ctx.scratch_zero("ssm_arrived", (ctx.runtime.max_requests,), torch.int32))
            self.out.run(ctx, x, accumulate)
            return
        dt = ctx.scratch("ssm_dt", (cap, self.heads), torch.float32)[:t]
        decay = ctx.scratch("ssm_decay", (cap, self.heads), torch.float32)[:t]
        pitch = -(-self.channels // 8) * 8
        # (workspaces sized once, for the largest step the runtime takes)
        n = ops.dscan_max_segments(max(ctx.runtime.max_batched_tokens, ctx.layout.t_cap),
                                   max(ctx.runtime.max_requests, requests))
        big = (n, self.heads, self.vdim, self.state_dim)
        own = ctx.scratch("ssm_seg_own", big, torch.float32)
        seg_decay = ctx.scratch("ssm_seg_decay", (n, self.heads), torch.float32)
        if self.chunks_ok:
            xbc = ctx.scratch("ssm_xbc", (cap, pitch), torch.bfloat16)[:t]
            kernels.prepare(xbc, dt, decay, as_log=True)
            kernels.chunks(xbc, dt, decay, own, ctx.scratch("ssm_seg_high", big, torch.bfloat16),
                           ctx.scratch("ssm_seg_low", big, torch.bfloat16), seg_decay)
        else:
            xbc = ctx.scratch("ssm_xbc", (cap, pitch), torch.float32)[:t]
            kernels.prepare(xbc, dt, decay, as_log=False)
            b, c = self.inner, self.inner + self.groups * self.state_dim
            share = self.heads // self.groups
            ops.decayed_scan(raw, xbc[:, c:self.channels], xbc[:, b:c], xbc[:, :b], decay, state,
                             ctx.q_start, ctx.state_slot, ctx.positions, requests, self.heads,
                             self.state_dim, self.vdim,
                             (own, ctx.scratch("ssm_seg_start", big, torch.float32), seg_decay),
                             share=(share, share), k_scale=dt, direct=self.direct, status=ctx.status)
        kernels.finish(gated=self.chunks_ok)
        self.out.run(ctx, x, accumulate)


register_part("mixer", "state_space", lambda p, store, rt: StateSpace(p, store, rt))
