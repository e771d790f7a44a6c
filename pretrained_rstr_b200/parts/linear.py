"""A linear map y = act(a . W^T + b) (+ residual): the building block of mixers,
feed-forwards and the head.

Weights are kept ``[out, in]`` with the input dimension contiguous, whatever layout
the checkpoint uses (GPT-2 stores Conv1D ``[in, out]``; the reference transposes it at
load time too, ``dev/examples/gpt2.clj:27-36``), in the runtime's element type.
Biases stay float32: they are added to the 32-bit accumulator.

float32 runtime: the true 32-bit FMA kernel.  bfloat16 runtime: the tensor-core
kernel with its fused epilogue.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..csrc import ops


class Linear:
    def __init__(self, weight: torch.Tensor, bias: Optional[torch.Tensor], runtime):
        if weight.dim() != 2:
            raise ValueError("Linear weight must be [out, in]")
        self.weight = weight.to(runtime.dtype).contiguous()
        self.bias = None if bias is None else bias.to(torch.float32).contiguous()
        self.n_out, self.n_in = self.weight.shape
        self.runtime = runtime
        if runtime.dtype != torch.float32 and self.n_in % 8 != 0:
            # the tensor-core kernels read rows in 16-byte pieces; said here, when the model
            # is built, rather than by the first step
            raise ValueError(f"a {str(runtime.dtype).replace('torch.', '')} product needs an input "
                             f"width that is a multiple of 8; this one has {self.n_in} "
                             f"(float32 takes any width)")

    @classmethod
    def from_store(cls, store, name: str, layout: str, n_in: int, n_out: int, bias: bool,
                   runtime) -> "Linear":
        w = store.get(name + ".weight")
        if layout == "in_out":
            if tuple(w.shape) != (n_in, n_out):
                raise ValueError(f"{name}.weight: expected [{n_in}, {n_out}], found {list(w.shape)}")
            w = w.to(runtime.dtype).t().contiguous()
        elif layout == "out_in":
            if tuple(w.shape) != (n_out, n_in):
                raise ValueError(f"{name}.weight: expected [{n_out}, {n_in}], found {list(w.shape)}")
        else:
            raise ValueError(f"unknown weight layout {layout!r}")
        b = store.get(name + ".bias") if bias else None
        return cls(w, b, runtime)

    def forward(self, ctx, a, out: torch.Tensor, act: Optional[str] = None,
                resid: Optional[torch.Tensor] = None, kv_scatter=None) -> bool:
        """out = act(a . W^T + bias) (+ resid).  ``out`` may be float32 (then ``resid`` may
        alias it) or the activation type.  ``a`` is a tensor, or a :class:`LazyNorm`: a
        norm that has not run yet, which the decode-time kernel computes in its prologue
        and every other kernel asks to run first.  ``kv_scatter`` = (k_pages, v_pages, slots,
        q_width[, only_cache]) offers the kernel the chance to write the key and value columns of a fused
        QKV product straight to the cache; returns True when it did."""
        m = out.shape[0]
        if self.runtime.dtype == torch.float32:
            ops.gemm_f32(out, _tensor(a), self.weight, self.bias, resid, act)
            return False
        # Which kernel (measured on GPT-2 small and XL shapes): up to 16 rows
        # the weight-streaming kernel with the norm fused into it; 17 to 64 rows the cluster
        # split-K kernel for narrow outputs and long reductions, the tensor-memory kernel for
        # wide outputs (the register-streaming kernel where K is no multiple of 64); beyond
        # 64 rows the tensor-memory kernel.
        max_rows, max_norm = ops.smallm_limits()
        if 16 < m <= 64 and (self.n_out <= 2048 or self.n_in >= 4 * self.n_out) and \
                ops.midm_supports(m, self.n_out, self.n_in):
            # narrow outputs or long reductions at a few dozen rows: the reduction split over
            # a thread-block cluster (measured against the other two kernels)
            ops.gemm_midm(out, _tensor(a), self.weight, self.bias, resid, act, status=ctx.status)
            return False
        if m <= max_rows and self.n_in % 8 == 0 and (m <= 16 or self.n_out <= 1024):
            if kv_scatter is not None and kv_scatter[0].dtype != out.dtype:
                kv_scatter = None
            if m <= 16 and isinstance(a, LazyNorm) and a.fusable and self.n_in <= max_norm:
                ops.gemm_smallm(out, self.weight, norm_input=a.x, gamma=a.norm.gamma,
                                beta=a.norm.beta, eps=a.norm.eps, bias=self.bias, resid=resid,
                                act=act, kv_scatter=kv_scatter, status=ctx.status,
                                norm_rows=a.rows, centred=getattr(a.norm, "centred", True))
            else:
                ops.gemm_smallm(out, self.weight, a=_tensor(a), bias=self.bias, resid=resid,
                                act=act, kv_scatter=kv_scatter, status=ctx.status)
            return kv_scatter is not None
        if kv_scatter is not None and (kv_scatter[0].dtype != out.dtype or resid is not None or
                                       kv_scatter[0].shape[3] % 8 != 0 or kv_scatter[3] % 8 != 0):
            kv_scatter = None
        ops.gemm_bf16(out, _tensor(a), self.weight, self.bias, resid, act, status=ctx.status,
                      kv_scatter=kv_scatter)
        return kv_scatter is not None


def padded_linear(weight: torch.Tensor, runtime) -> Linear:
    """A Linear over ``weight`` [out, in] whose input width is rounded up to a multiple of 8
    with zero columns (what the tensor-core kernels read in 16-byte pieces).  The caller keeps
    its input in a buffer of ``n_in`` columns from ``ctx.scratch_zero`` and writes the real
    columns only: the rest stay zero."""
    k = weight.shape[1]
    k_pad = -(-k // 8) * 8
    if k_pad != k:
        weight = torch.cat([weight, torch.zeros((weight.shape[0], k_pad - k), dtype=weight.dtype,
                                                device=weight.device)], dim=1)
    return Linear(weight, None, runtime)


class ResultProduct:
    """The matrix product a part ends with: x (+)= r . W^T + b, from a buffer of its own that the
    part fills (:meth:`buffer`, then :meth:`run`).

    Results that join the same stream can share one product: ``a.absorb(b)`` puts b's matrix beside
    a's (a row of the common buffer is [r_a | r_b]; biases add up), ``b.run`` then does nothing, and
    whoever joined them sets ``a.closer`` and calls :meth:`close` when all have filled their
    columns.  Segments start at multiples of 8 columns; the columns between stay zero."""

    def __init__(self, weight: torch.Tensor, runtime, key: str, bias: Optional[torch.Tensor] = None):
        self.runtime, self.key = runtime, key
        self.n_out = int(weight.shape[0])
        self.parts = [(weight, bias)]
        self.host: Optional["ResultProduct"] = None
        self.column = 0                        # first column in the common buffer
        self.columns = -(-int(weight.shape[1]) // 8) * 8
        self.total = self.columns              # (of all that share the product)
        self.closer = None                     # who runs the common product, or None: run() does
        self._linear: Optional[Linear] = None

    def absorb(self, other: "ResultProduct") -> None:
        if other is self or self.host is not None or other.host is not None or \
                self._linear is not None or other._linear is not None:
            raise RuntimeError("result products can be joined once, before they are built")
        if other.n_out != self.n_out:
            raise ValueError(f"result products of {self.n_out} and {other.n_out} outputs")
        for guest in [other] + getattr(other, "guests", []):
            guest.host = self
            guest.column += self.total
        self.guests = getattr(self, "guests", []) + [other] + getattr(other, "guests", [])
        self.parts += other.parts
        self.key = f"{self.key}+{other.key}"
        self.total += other.total
        other.parts = []

    def linear(self) -> Linear:
        if self._linear is None:
            pieces, bias = [], None
            for w, b in self.parts:
                pieces.append(w.to(self.runtime.dtype))
                pad = -w.shape[1] % 8
                if pad:
                    pieces.append(torch.zeros((w.shape[0], pad), dtype=self.runtime.dtype, device=w.device))
                if b is not None:
                    bias = b.to(torch.float32) if bias is None else bias + b.to(torch.float32)
            # (the buffer's layout is part of its name: columns that stay zero lie elsewhere in another)
            self.key += "/" + ",".join(str(int(w.shape[1])) for w, _b in self.parts)
            self._linear = Linear(torch.cat(pieces, dim=1) if len(pieces) > 1 else pieces[0], bias,
                                  self.runtime)
            self.parts = []
        return self._linear

    def buffer(self, ctx, t: int) -> torch.Tensor:
        """[t, columns] in the activation type: the part writes its real columns."""
        host = self.host or self
        host.linear()
        rows = ctx.scratch_zero(host.key, (ctx.token_capacity, host.total), self.runtime.dtype)[:t]
        return rows if host.total == self.columns else rows[:, self.column:self.column + self.columns]

    def run(self, ctx, x: torch.Tensor, accumulate: bool = True) -> None:
        if self.host is None and self.closer is None:
            self.close(ctx, x, accumulate)

    def close(self, ctx, x: torch.Tensor, accumulate: bool = True) -> None:
        if self.host is not None:
            return
        lin = self.linear()
        rows = ctx.scratch_zero(self.key, (ctx.token_capacity, self.total), self.runtime.dtype)[:x.shape[0]]
        lin.forward(ctx, rows, x, resid=x if accumulate else None)


class LazyNorm:
    """A norm of ``x`` (of its rows ``rows``, if given: an int32 tensor of row indices) that
    runs when its result is first needed.  A consumer that can compute the norm itself
    (``fusable``: a plain layer norm, or a root-mean-square norm that is a weight per coordinate
    times x / rms(x)) reads ``x``, ``rows`` and ``norm`` instead and the norm
    never runs as a kernel of its own."""

    def __init__(self, ctx, norm, x: torch.Tensor, out: torch.Tensor, rows=None):
        self.ctx, self.norm, self.x, self._out, self.rows = ctx, norm, x, out, rows
        self._done = False
        # (a layer norm, or a root-mean-square norm with a weight per coordinate and no other
        # factor: the same prologue without the mean)
        self.fusable = all(hasattr(norm, f) for f in ("gamma", "beta", "eps")) and \
            getattr(norm, "kind", "") in ("layer_norm", "rms_norm") and norm.gamma is not None
        self.shape = out.shape

    @property
    def done(self) -> bool:
        return self._done

    def tensor(self) -> torch.Tensor:
        if not self._done:
            if self.rows is None:
                self.norm.forward(self.ctx, self.x, self._out)
            else:
                self.norm.forward(self.ctx, self.x, self._out, rows=self.rows)
            self._done = True
        return self._out


def _tensor(a) -> torch.Tensor:
    return a.tensor() if isinstance(a, LazyNorm) else a
