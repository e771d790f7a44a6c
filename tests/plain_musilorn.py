"""A plain, slow implementation of the Musilorn design in float64 on the CPU: one function per
mechanism, written from the design's equations, with its own reader of model folders.  It
shares no code with the package; the GPU tests compare the engine with it.

Notation: T tokens of one sequence at positions 0..T-1; x the residual stream [T, width];
matrices are stored [out, in] and applied as ``h @ W.T``.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional

import numpy as np
import torch

F64 = torch.float64


# ----------------------------------------------------------------------- model folders
def read_folder(folder: str):
    """(config dict, {name: float64 tensor}) of a folder with config.json and
    model.safetensors (8-byte little-endian header length, a JSON header, the data)."""
    with open(os.path.join(folder, "config.json"), "r", encoding="utf-8") as fh:
        cfg = json.load(fh)
    with open(os.path.join(folder, "model.safetensors"), "rb") as fh:
        (n,) = struct.unpack("<Q", fh.read(8))
        header = json.loads(fh.read(n))
        blob = fh.read()
    tensors = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        raw = blob[lo:hi]
        if meta["dtype"] == "BF16":
            bits = np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16
            t = torch.from_numpy(bits.view(np.float32).copy()).to(F64)
        elif meta["dtype"] == "F32":
            t = torch.from_numpy(np.frombuffer(raw, dtype="<f4").copy()).to(F64)
        else:
            raise ValueError(f"{name}: element type {meta['dtype']}")
        tensors[name] = t.reshape(meta["shape"])
    return cfg, tensors


# ---------------------------------------------------------------------------------- norms
def unit_rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    """v / sqrt(mean(v^2) + eps) over the last axis."""
    return v / torch.sqrt(v.pow(2).mean(dim=-1, keepdim=True) + eps)


def centred_norm(v: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    """(v - mean) / sqrt(variance + eps) * w + b, the variance over all coordinates."""
    c = v - v.mean(dim=-1, keepdim=True)
    return c / torch.sqrt(c.pow(2).mean(dim=-1, keepdim=True) + eps) * w + b


# ------------------------------------------------------------------------------ rotations
def plain_frequencies(base: float, dims: int) -> List[float]:
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def banded_frequencies(freqs: List[float], factor: float, low: float, high: float,
                       original: float) -> List[float]:
    """Frequencies by their wavelength: short ones stay, long ones are divided by ``factor``,
    the band between blends the two."""
    out = []
    for f in freqs:
        wavelength = 2.0 * math.pi / f
        if wavelength < original / high:
            out.append(f)
        elif wavelength > original / low:
            out.append(f / factor)
        else:
            s = (original / wavelength - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return out


def turn(v: torch.Tensor, positions: torch.Tensor, freqs: List[float], layout: str) -> torch.Tensor:
    """v [T, heads, n]: the first 2 * len(freqs) coordinates of every head turned by position x
    frequency; pairs (i, i + dims / 2) in the "half" layout, (2i, 2i + 1) in "interleaved"."""
    dims = 2 * len(freqs)
    if dims == 0:
        return v
    angle = positions.to(F64)[:, None, None] * torch.tensor(freqs, dtype=F64)[None, None, :]
    c, s = torch.cos(angle), torch.sin(angle)
    out = v.clone()
    if layout == "half":
        first, second = slice(0, dims // 2), slice(dims // 2, dims)
    else:
        first, second = slice(0, dims, 2), slice(1, dims, 2)
    a, b = v[..., first], v[..., second]
    out[..., first] = a * c - b * s
    out[..., second] = b * c + a * s
    return out


# ------------------------------------------------------------------------------ attention
def causal_convolution(u: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """u [T, C], taps [C, n] (the last column is the current token's), zeros before the start."""
    T, n = u.shape[0], taps.shape[1]
    out = torch.zeros_like(u)
    for j in range(n):
        back = n - 1 - j
        if back < T:
            out[back:] += taps[:, j] * u[:T - back]
    return out


def capped_sink_attention(q, k, v, scale: float, cap: Optional[float], sink: bool = True) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V], causal; query head h uses key/value
    head h // (H / G); scores pass cap * tanh(. / cap); the denominator has 1 added (a key of
    score 0 without a value)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    hidden = torch.triu(torch.ones(T, T, dtype=torch.bool), diagonal=1)
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        s = s.masked_fill(hidden, -math.inf)
        top = s.max(dim=-1, keepdim=True).values.clamp(min=0.0)
        e = torch.exp(s - top)
        total = e.sum(dim=-1, keepdim=True)
        if sink:
            total = total + torch.exp(-top)
        out[:, h] = (e / total) @ v[:, h // per]
    return out


def _exact(v: torch.Tensor) -> torch.Tensor:
    return v


def attention_mixer(W, p: str, mx: dict, h: torch.Tensor, positions, eps: float,
                    r=_exact) -> torch.Tensor:
    """Queries and keys behind a short convolution; the convolved keys are the values; then a
    norm per head with a shared weight, the rotation of interleaved pairs, the attention.  ``r``:
    a rounding of what is cached and of what the output product reads."""
    T = h.shape[0]
    H, G, D = mx["heads"], mx["kv_heads"], mx["dim"]
    q = causal_convolution(h @ W[p + "q"].T, W[p + "q.conv"]).reshape(T, H, D)
    k = causal_convolution(h @ W[p + "k"].T, W[p + "k.conv"]).reshape(T, G, D)
    v = k
    q = unit_rms(q, eps) * W[p + "q.norm"]
    k = unit_rms(k, eps) * W[p + "k.norm"]
    freqs = plain_frequencies(mx["rot"]["base"], mx["rot"]["dims"])
    sc = mx["rot"].get("scaling")
    if sc:
        freqs = banded_frequencies(freqs, sc["factor"], sc["low"], sc["high"], sc["original"])
    q, k = turn(q, positions, freqs, "interleaved"), turn(k, positions, freqs, "interleaved")
    o = capped_sink_attention(q, r(k), r(v), mx["scale"], mx.get("softcap"))
    return r(o.reshape(T, H * D)) @ W[p + "o"].T


# ------------------------------------------------------------------------------ retention
def retention_outputs(q, k, v, decay: List[float]) -> torch.Tensor:
    """q, k [T, H, D], v [T, H, V]: S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F64)
    d = torch.tensor(decay, dtype=F64)[:, None, None]
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def retention_mixer(W, p: str, mx: dict, h, positions, eps: float, r=_exact) -> torch.Tensor:
    T = h.shape[0]
    H, D, V = mx["heads"], mx["dim"], mx["vdim"]
    q, k = (h @ W[p + "q"].T).reshape(T, H, D), (h @ W[p + "k"].T).reshape(T, H, D)
    v = (h @ W[p + "v"].T).reshape(T, H, V)
    freqs = plain_frequencies(mx["rot"]["base"], mx["rot"]["dims"])
    q = turn(q, positions, freqs, "half")
    k = turn(k, positions, freqs, "half") * D ** -0.5
    o = unit_rms(retention_outputs(q, k, v, mx["decay"]), eps).reshape(T, H * V)
    return r(o * torch.nn.functional.silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------------------- the rest
def tanh_gelu(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z.pow(3))))


def gated_unit(W, p: str, h, r=_exact) -> torch.Tensor:
    return r(tanh_gelu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def run_list(cfg: dict):
    """(layer, first of a pass) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(a)]
    for _ in range(loop["times"]):
        runs += [(i, i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def _bf16(x: torch.Tensor) -> torch.Tensor:
    return x.to(torch.float32).to(torch.bfloat16).to(F64)


def forward(tokens: List[int], W: Dict[str, torch.Tensor], cfg: dict,
            taps: Optional[list] = None, rounded: bool = False) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``taps`` collects the stream after every layer run.
    ``rounded``: what the matrix products read (norms of the stream, the stream where a pass
    begins, mixers' results, activations) and what is cached is rounded to bfloat16, as serving in
    bfloat16 does; the difference to the exact run says how far rounding alone moves a row."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    r = _bf16 if rounded else _exact
    norm = lambda v, name: centred_norm(v, W[name], W[name + ".b"], eps)
    positions = torch.arange(len(tokens))
    x0 = W["embed"][tokens]
    x = x0
    for i, first in run_list(cfg):
        if first:
            x = r(torch.cat([x, x0], dim=-1)) @ W["loop.in"].T
        layer, p = cfg["layers"][i], f"l{i}."
        mixer = attention_mixer if layer["type"] == "attention" else retention_mixer
        y = mixer(W, p + "mix.", layer["mixer"], r(norm(x, p + "norm1")), positions, eps, r)
        x = x + m * norm(y, p + "norm1b")
        if layer.get("mlp"):
            x = x + m * norm(gated_unit(W, p + "mlp.", r(norm(x, p + "norm2")), r), p + "norm2b")
        if taps is not None:
            taps.append(x.clone())
    logits = r(norm(x, "final.norm")) @ W["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits


def greedy(prompt: List[int], n_new: int, W: Dict[str, torch.Tensor], cfg: dict) -> List[int]:
    """The ``n_new`` tokens greedy decoding appends (the whole sequence runs again per token)."""
    ids, out = list(prompt), []
    for _ in range(n_new):
        nxt = int(forward(ids, W, cfg)[-1].argmax())
        out.append(nxt)
        ids.append(nxt)
    return out
