"""Softmax attention over the paged cache with the options of windowed designs, as a mixer.

Query head h uses key/value head h // (heads / kv_heads); keys have ``dim`` numbers a head,
values ``vdim``.  Every option is a parameter, and a design names the ones it has:

``window`` / ``keep_first``  position i sees j <= i with i - j < window, or j < keep_first (the
                      sequence's first tokens stay visible at their true positions); window
                      None or 0: every earlier key
``rot_dims`` / ``rot_base``  rotary positions on each head's first coordinates; ``rot_layout`` "half"
                      or "interleaved" (pairs (2i, 2i + 1)); ``rot_factor``: every frequency is
                      divided by it (linear scaling); ``rot_bands`` {factor, low, high, original}:
                      frequencies scaled by their wavelength (see ``banded_frequencies``);
                      ``rot_yarn`` {factor, original, fast, slow}: YaRN's frequencies, with its
                      magnitude on cosines and sines (see ``yarn_frequencies``)
``conv``              a causal convolution over time on every channel of q and k, ``conv`` taps
                      long, without a bias (weights ``q_conv`` / ``k_conv``, [channels, taps]), before
                      norm and rotation.  The last taps - 1 projected values of a request are
                      per-request STATE (32-bit, a slot per live request)
``keys_are_values``   no value projection: a key as it is before norm and rotation is its value
``softcap``           scores are softcap * tanh(score / softcap)
``qk_norm``           a root-mean-square norm over the whole query projection and over the
                      whole key projection before they are split into heads (weights
                      ``q_norm`` / ``k_norm``); "head": per head, before the rotation, with
                      weights of ``dim`` numbers that all heads share; "head_after": per head,
                      after the rotation, without weights
``bias``              q, k and v have biases (weights ``q_bias`` / ``k_bias`` / ``v_bias``);
                      ``out_bias``: so has the output projection (weight ``out_bias``)
``sink``              a learned number per head (weight ``sink``) whose exponential joins the
                      softmax's denominator once: it has no key and no value and is not scaled;
                      ``sink_score``: the same with one constant for all heads (0: the
                      denominator has 1 added)
``q_temp``            (coef, every): queries are multiplied by 1 + coef * ln(floor((p + 1) /
                      every) + 1) at position p
``slope_bits``        a distance bias slope_h * (i - j) is taken off the scores, slope_h =
                      2^(-slope_bits * (h + 1) / heads); None: no bias
``head_gate``         head h's result is multiplied by sigmoid(G x)_h (weight ``gate``, one
                      row a head; it rides in the first product)
``value_gate``        the concatenated heads are multiplied element by element by sigmoid(G x)
                      (weight ``gate``, heads * vdim rows; in the first product too)
``out_scale``         a constant on the result (a mixer that sums two mixers gives each one)
``shares_cache``      the layer has no key/value tensors: it attends over the cache rows
                      another layer wrote, with queries, mask and everything else of its own

The cache holds ONE row per (token, key/value head), [k | v] (a group with one pool per layer),
keys as the attention reads them (normed, rotated).  Q, K, V and the gate are one matrix
product whose 32-bit result is normed and rotated unrounded; scores, weights and sums are
32-bit.  Norms per head, biases, the convolution and interleaved pairs are one kernel of a warp per
(token, head), which reads its angles' cosines and sines from a table the step computes once.  Every key is kept: a window's pages are not given back, since kept first tokens and
layers that share a cache with another window may still read them.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .interfaces import KVSpec, LayerCache, Mixer, StateSpec
from .latent_attention import FusedInput
from .linear import ResultProduct
from .positions_rotary import (RotaryAngles, banded_frequencies, rotary_frequencies,
                               split_frequencies, yarn_frequencies)
from .registry import register_part


class WindowAttention(Mixer):
    graph_safe = True
    can_overwrite = True
    accepts_lazy_norm = True      # the first matrix product may compute the norm itself

    def __init__(self, p: dict, store, runtime):
        w = p["weights"]
        self.width, self.heads, self.kv_heads = int(p["width"]), int(p["heads"]), int(p["kv_heads"])
        self.dim, self.vdim = int(p["dim"]), int(p["vdim"])
        self.scale, self.eps = float(p["scale"]), float(p.get("eps", 0.0))
        self.window, self.keep_first = int(p.get("window") or 0), int(p.get("keep_first") or 0)
        self.rot_dims = int(p.get("rot_dims") or 0)
        self.out_scale = float(p.get("out_scale", 1.0))
        self.shares_cache = bool(p.get("shares_cache", False))
        self.keys_are_values = bool(p.get("keys_are_values", False))
        self.taps = int(p.get("conv") or 0)
        self.softcap = float(p.get("softcap") or 0.0)
        self.interleaved = {"half": False, "interleaved": True}[p.get("rot_layout", "half")]
        temp = p.get("q_temp")
        self.temp_coef, self.temp_every = (float(temp[0]), int(temp[1])) if temp else (0.0, 0)
        self.runtime = runtime
        if self.heads % self.kv_heads:
            raise ValueError(f"window_attention: {self.heads} query heads are not a multiple of "
                             f"{self.kv_heads} key/value heads")
        if self.rot_dims % 2 or self.rot_dims > self.dim:
            raise ValueError(f"window_attention: {self.rot_dims} rotated coordinates of {self.dim}")
        if self.vdim > 512:
            raise ValueError("window_attention: value heads wider than 512 are not built")
        if self.keys_are_values and self.vdim != self.dim:
            raise ValueError(f"window_attention: keys of {self.dim} numbers cannot be values of {self.vdim}")
        if self.softcap < 0.0 or self.taps < 0:
            raise ValueError("window_attention: a cap and a convolution's taps cannot be negative")
        if self.shares_cache and (self.taps or self.keys_are_values):
            raise ValueError("window_attention: a layer that reads another layer's cache has neither a "
                             "convolution nor keys as values")
        if temp and self.temp_every < 1:
            raise ValueError("window_attention: the query temperature's period must be positive")

        def need(name, shape):
            t = store.get(w[name])
            if tuple(t.shape) != tuple(shape):
                raise ValueError(f"{w[name]}: expected {list(shape)}, found {list(t.shape)}")
            return t

        dev = runtime.device
        self.input = FusedInput(self.width, runtime, "wattn_in")
        self.input.add("q", need("q", (self.heads * self.dim, self.width)))
        if not self.shares_cache:
            self.input.add("k", need("k", (self.kv_heads * self.dim, self.width)))
            if not self.keys_are_values:
                self.input.add("v", need("v", (self.kv_heads * self.vdim, self.width)))
        self.value_gate = bool(p.get("value_gate"))
        self.gated = bool(p.get("head_gate")) or self.value_gate
        if self.gated:
            rows = self.heads * self.vdim if self.value_gate else self.heads
            self.input.add("gate", need("gate", (rows, self.width)))
        self.q_norm = self.k_norm = None
        mode = p.get("qk_norm")
        if mode not in (None, False, True, "whole", "head", "head_after"):
            raise ValueError(f"window_attention: unknown qk_norm {mode!r}")
        self.head_norm = {"head": "before", "head_after": "after"}.get(mode)
        if mode == "head":
            self.q_norm = need("q_norm", (self.dim,)).to(torch.float32).contiguous()
            if not self.shares_cache:
                self.k_norm = need("k_norm", (self.dim,)).to(torch.float32).contiguous()
        elif mode in (True, "whole"):
            self.q_norm = need("q_norm", (self.heads * self.dim,)).to(torch.float32).contiguous()
            if not self.shares_cache:
                self.k_norm = need("k_norm", (self.kv_heads * self.dim,)).to(torch.float32).contiguous()
        self.biases = None
        if p.get("bias"):
            f32 = lambda t: t.to(torch.float32).contiguous()
            self.biases = (f32(need("q_bias", (self.heads * self.dim,))),
                           None if self.shares_cache else f32(need("k_bias", (self.kv_heads * self.dim,))),
                           None if self.shares_cache else f32(need("v_bias", (self.kv_heads * self.vdim,))))
        self.sinks = need("sink", (self.heads,)).to(torch.float32).contiguous() if p.get("sink") else None
        if p.get("sink_score") is not None:
            if self.sinks is not None:
                raise ValueError("window_attention: either a learned sink or a constant one")
            self.sinks = torch.full((self.heads,), float(p["sink_score"]), dtype=torch.float32, device=dev)
        self.conv_w = None
        if self.taps:
            self.conv_w = tuple(need(n, (h * self.dim, self.taps)).to(torch.float32).contiguous()
                                for n, h in (("q_conv", self.heads), ("k_conv", self.kv_heads)))
        out_bias = None
        if p.get("out_bias"):              # (the mixer's constant acts on the bias too)
            out_bias = need("out_bias", (self.width,)).to(torch.float32) * self.out_scale
        self.out = ResultProduct(need("out", (self.width, self.heads * self.vdim)), runtime, "wattn_out",
                                 out_bias)
        self.slopes = None
        if p.get("slope_bits") is not None:
            bits = float(p["slope_bits"])
            self.slopes = torch.tensor([2.0 ** (-bits * (h + 1) / self.heads)
                                        for h in range(self.heads)],
                                       dtype=torch.float64).to(torch.float32).to(dev)
        base, bands = float(p.get("rot_base", 10000.0)), p.get("rot_bands")
        yarn, magnitude = p.get("rot_yarn"), 1.0
        if yarn and mode in (True, "whole"):
            raise ValueError("window_attention: a norm over whole projections goes with no stretched angles")
        if yarn and self.rot_dims:
            (self.freq, self.freq_lo), magnitude = yarn_frequencies(
                base, self.rot_dims, float(yarn["factor"]), float(yarn["original"]), float(yarn["fast"]),
                float(yarn["slow"]), dev, with_lo=True)
        elif bands and self.rot_dims:
            self.freq, self.freq_lo = split_frequencies(
                banded_frequencies(base, self.rot_dims, float(bands["factor"]), float(bands["low"]),
                                   float(bands["high"]), float(bands["original"])), dev)
        else:
            self.freq, self.freq_lo = rotary_frequencies(
                base, self.rot_dims, dev, divide_by=float(p.get("rot_factor") or 1.0), with_lo=True)
        # (a norm over whole projections is another kernel, which computes its own angles)
        self.rotary = RotaryAngles(self.freq, self.freq_lo, magnitude) \
            if self.rot_dims and mode not in (True, "whole") else None
        gpu = torch.cuda.is_available()
        # kernels for bfloat16 cache rows: (portions, single tokens)
        self.bf16_ok = ops.wattn_bf16_supports(self.heads, self.kv_heads, self.dim, self.vdim) \
            if gpu and runtime.dtype == torch.bfloat16 else (False, False)
        self.tile_rows = ops.wattn_tile_rows(self.heads, self.kv_heads, self.dim, self.vdim) if gpu else 0
        self.single_ok = gpu and ops.wattn_single_supports(self.heads, self.kv_heads, self.dim, self.vdim)

    def kv_spec(self) -> KVSpec:
        return KVSpec(self.kv_heads, self.dim + self.vdim, None, values=False)

    def state_specs(self):
        if not self.taps:
            return []
        return [StateSpec("attention_conv", (self.taps - 1, (self.heads + self.kv_heads) * self.dim),
                          torch.float32)]

    def step_bytes(self, context: int) -> int:
        """Bytes a single token at ``context`` tokens reads: the rows it sees, its saved inputs."""
        seen = min(context, self.window + self.keep_first) if self.window else context
        rows = seen * self.kv_heads * (self.dim + self.vdim) * self.runtime.dtype.itemsize
        inputs = max(self.taps - 1, 0) * (self.heads + self.kv_heads) * self.dim
        return rows + 2 * 4 * inputs                 # (a convolution's saved inputs: read, written back)

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

    def forward(self, ctx, h, x, cache: LayerCache, accumulate: bool = True) -> None:
        if self.shares_cache == cache.writes:
            raise ValueError("window_attention: a layer without key/value tensors reads another "
                             "layer's cache, and only such a layer does")
        t = x.shape[0]
        cap = ctx.token_capacity
        group = ctx.groups[cache.group]
        proj = self._proj = self.input.run(ctx, h)
        cols = self.input.cols
        q = ctx.scratch("wattn_q", (cap, self.heads * self.dim), torch.float32)[:t]
        conv = None
        if self.taps:
            # (a step in which every request brings one token: the same kernel brings the
            # convolution's saved inputs up to date)
            conv = (*self.conv_w, cache.state["attention_conv"], ctx.seq_of_token, ctx.q_start,
                    ctx.state_slot, 0 if ctx.max_q_len == 1 else ctx.layout.b_cap)
        ops.wattn_prepare(q, cache.k, proj, cols["q"][0],
                          0 if self.shares_cache else cols["k"][0],
                          0 if self.shares_cache or self.keys_are_values else cols["v"][0],
                          self.q_norm, self.k_norm,
                          None if self.shares_cache else group.slots, ctx.positions, self.freq,
                          self.heads, self.kv_heads, self.dim, self.vdim, self.rot_dims, self.eps,
                          self.temp_coef, self.temp_every, ctx.status, head_norm=self.head_norm,
                          biases=self.biases, freq_lo=self.freq_lo,
                          angles=self.rotary.table(ctx, t) if self.rotary else None,
                          interleaved=self.interleaved, keys_are_values=self.keys_are_values,
                          conv=conv)
        o = self.out.buffer(ctx, t)
        # a step of single tokens: a CTA per (token, key/value head) whose warps share out the
        # key blocks (rows of different requests share no keys); sizes that kernel does not
        # take: the tiled kernel, a row a CTA.  Serving in bfloat16 has kernels of its own for
        # both kinds of step
        single = ctx.max_q_len == 1 or ctx.layout.t_cap <= ctx.layout.b_cap
        ops.wattn(o, q, cache.k, group.block_table, ctx.seq_of_token, ctx.positions, self.heads,
                  self.dim, self.vdim, self.window, self.keep_first, self.scale,
                  gate=proj[:, cols["gate"][0]:] if self.gated else None, slopes=self.slopes,
                  out_scale=self.out_scale, status=ctx.status,
                  tile_rows=min(self.tile_rows, 1) if single else self.tile_rows,
                  single=single and self.single_ok, sinks=self.sinks,
                  gate_per_value=self.value_gate, softcap=self.softcap,
                  bf16_kernels=self.bf16_ok[1 if single else 0])
        self.out.run(ctx, x, accumulate)


register_part("mixer", "window_attention", lambda p, store, rt: WindowAttention(p, store, rt))
