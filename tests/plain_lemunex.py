"""A plain, slow implementation of the Lemunex design in float64 on the CPU: one function per
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
        if meta["dtype"] == "BF16":
            bits = np.frombuffer(blob[lo:hi], dtype="<u2").astype(np.uint32) << 16
            t = torch.from_numpy(bits.view(np.float32).copy())
        elif meta["dtype"] == "F32":
            t = torch.from_numpy(np.frombuffer(blob[lo:hi], dtype="<f4").copy())
        else:
            raise ValueError(f"{name}: element type {meta['dtype']}")
        tensors[name] = t.to(F64).reshape(meta["shape"])
    return cfg, tensors


# -------------------------------------------------------------------------- small pieces
def unit_rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    """v / sqrt(mean(v^2) + eps) over the last axis."""
    return v / torch.sqrt(v.pow(2).mean(dim=-1, keepdim=True) + eps)


def offset_norm(v: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """A norm whose weight is stored around zero: unit_rms(v) * (1 + w)."""
    return unit_rms(v, eps) * (1.0 + w)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def log1p_exp(z: torch.Tensor) -> torch.Tensor:
    """softplus without a threshold."""
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def exact(t: torch.Tensor) -> torch.Tensor:
    return t


def to_bfloat16(t: torch.Tensor) -> torch.Tensor:
    """What storing ``t`` in bfloat16 leaves of it.  Mixers and feed-forwards take ``r``: ``exact``, or
    this, applied to what serving in bfloat16 stores between two products."""
    return t.to(torch.bfloat16).to(F64)


# ----------------------------------------------------------------------------- attention
def angle_table(rot: dict):
    """(frequencies, magnitude).  Without ``scaling``: base^(-2i/dims), 1.  With it, pair i keeps
    its frequency where it turns fast and has it divided by the factor where it turns slowly, a
    linear ramp between, and both sides of a score are stretched by the magnitude."""
    dims, base = rot["dims"], rot["base"]
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(plain, dtype=F64), 1.0

    def pair_of(turns: float) -> float:
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_of(sc["fast"])), 0)
    hi = min(math.ceil(pair_of(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1.0 - ramp))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(sc["factor"]) + 1.0


def turn_pairs(v: torch.Tensor, positions: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """v [T, heads, n]: pairs (2i, 2i + 1) of the first ``dims`` coordinates turned by position x
    frequency i and stretched by the magnitude."""
    if not rot or rot["dims"] == 0:
        return v
    freq, mag = angle_table(rot)
    dims = rot["dims"]
    angle = positions.to(F64)[:, None, None] * freq[None, None, :]
    c, s = torch.cos(angle) * mag, torch.sin(angle) * mag
    a, b = v[..., 0:dims:2], v[..., 1:dims:2]
    out = v.clone()
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def sliding_attention(q, k, v, scale: float, window: Optional[int]) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]: query head h uses key/value head
    h // (H / G); position i sees 0 <= i - j < window (None: every earlier one)."""
    T, H, _ = q.shape
    G = k.shape[1]
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    seen = back >= 0
    if window:
        seen = seen & (back < window)
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        score = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf)
        out[:, h] = torch.softmax(score, dim=-1) @ v[:, g]
    return out


def attention_mixer(W, p: str, mx: dict, h, positions, r=exact) -> torch.Tensor:
    """Biased projections, rotated queries and keys, a window, a gate per head, a biased output."""
    T = h.shape[0]
    H, G, D, V = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = (h @ W[p + "q"].T + W[p + "q.b"]).reshape(T, H, D)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).reshape(T, G, D)
    v = (h @ W[p + "v"].T + W[p + "v.b"]).reshape(T, G, V)
    q, k = turn_pairs(q, positions, mx.get("rot")), turn_pairs(k, positions, mx.get("rot"))
    o = sliding_attention(q, r(k), r(v), mx["scale"], (mx.get("mask") or {}).get("size"))
    o = o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return r(o).reshape(T, H * V) @ W[p + "o"].T + W[p + "o.b"]


# ---------------------------------------------------------------------- recurrent mixers
def decayed_memory(q, k, v, log_decay) -> torch.Tensor:
    """S_t = diag(exp(log_decay_t)) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head, from S = 0;
    q, k, log_decay [T, H, D], v [T, H, V] -> [T, H, V]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F64)
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        S = torch.exp(log_decay[t])[:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def gated_linear_mixer(W, p: str, mx: dict, h, eps: float, r=exact) -> torch.Tensor:
    T = h.shape[0]
    H, D, V = mx["heads"], mx["dim"], mx["vdim"]
    q = (h @ W[p + "q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ W[p + "k"].T).reshape(T, H, D)
    v = (h @ W[p + "v"].T).reshape(T, H, V)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    log_decay = (-log1p_exp(-z) / mx["tau"]).reshape(T, H, D)
    o = unit_rms(decayed_memory(q, k, v, log_decay), eps) * W[p + "norm"]
    return r(o.reshape(T, H * V) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def causal_convolution(x: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, n] (the last column is the current token's), zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    out = bias.expand(T, -1).clone()
    for j in range(n):
        back = n - 1 - j
        if back < T:
            out[back:] += taps[:, j] * x[:T - back]
    return out


def state_space_mixer(W, p: str, mx: dict, h, eps: float, r=exact) -> torch.Tensor:
    """A scalar decay per head and token, keys B and queries C shared by a group's heads, step
    sizes on the keys, a direct path D, the gate before a norm in equal parts."""
    T = h.shape[0]
    H, V, N, G = mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    inner = H * V
    z, xbc, dt = torch.split(h @ W[p + "in"].T, [inner, inner + 2 * G * N, H], dim=1)
    xbc = r(silu(causal_convolution(xbc, W[p + "conv"], W[p + "conv.b"])))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    x = x.reshape(T, H, V)
    B = B.reshape(T, G, N).repeat_interleave(H // G, dim=1)
    C = C.reshape(T, G, N).repeat_interleave(H // G, dim=1)
    dt = log1p_exp(dt + W[p + "dt_bias"])
    log_decay = (-torch.exp(W[p + "A_log"]) * dt)[:, :, None].expand(T, H, N)
    y = decayed_memory(C, B * dt[:, :, None], x, log_decay) + W[p + "D"][:, None] * x
    y = (y.reshape(T, inner) * silu(z)).reshape(T, mx["norm_groups"], -1)
    return r(unit_rms(y, eps).reshape(T, inner) * W[p + "norm"]) @ W[p + "o"].T


# ------------------------------------------------------------------------- feed-forwards
def gated_unit(W, p: str, h, r=exact) -> torch.Tensor:
    return r(silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def routed_unit(W, p: str, mlp: dict, h, margins: Optional[list] = None, r=exact) -> torch.Tensor:
    """Softmax scores over all experts; chosen by score + correction, weighted by the score
    alone; the last ``identity`` experts give back their input; a gated shared expert.
    ``margins`` collects how far the last chosen and the first unchosen expert lie apart [T]."""
    router = mlp["router"]
    real, top = router["experts"], router["top"]
    scores = torch.softmax(h @ W[p + "router"].T, dim=-1)
    choice = scores + W[p + "correction"]
    chosen = torch.topk(choice, top, dim=-1).indices
    if margins is not None and top < choice.shape[1]:
        ranked = choice.sort(dim=-1, descending=True).values
        margins.append(ranked[:, top - 1] - ranked[:, top])
    weight = torch.zeros_like(scores).scatter(1, chosen, scores.gather(1, chosen))
    out = weight[:, real:].sum(-1, keepdim=True) * h
    for e in range(real):
        out = out + weight[:, e:e + 1] * gated_unit(W, f"{p}e{e}.", h, r)
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ W[p + "shared.sg"].T) * gated_unit(W, p + "shared.", h, r)
    return out


def feed_forward(W, p: str, mlp: dict, h, margins: Optional[list] = None, r=exact) -> torch.Tensor:
    if mlp["kind"] == "dense":
        return r(torch.relu(h @ W[p + "up"].T).pow(2)) @ W[p + "down"].T
    return routed_unit(W, p, mlp, h, margins, r)


# ------------------------------------------------------------------------------ the model
def mixer(W, p: str, layer: dict, h, positions, eps: float, r=exact) -> torch.Tensor:
    mx = layer["mixer"]
    if layer["type"] == "mamba2":
        return state_space_mixer(W, p, mx, h, eps, r)
    return mx["left_scale"] * attention_mixer(W, p + "left.", mx["left"], h, positions, r) + \
        mx["right_scale"] * gated_linear_mixer(W, p + "right.", mx["right"], h, eps, r)


def forward(tokens: List[int], W: Dict[str, torch.Tensor], cfg: dict,
            taps: Optional[list] = None, rounded: bool = False,
            margins: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``taps`` collects the stream after every layer,
    ``margins`` the routers' margins (see ``routed_unit``).
    ``rounded``: what serving in bfloat16 stores between two products is rounded to it; the
    difference to the exact run says how far rounding alone moves a row."""
    eps = cfg["norm"]["eps"]
    r = to_bfloat16 if rounded else exact
    positions = torch.arange(len(tokens))
    x = offset_norm(W["embed"][tokens], W["embed.norm"], eps)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = r(offset_norm(x, W[p + "norm1"], eps))
        y = mixer(W, p + "mix.", layer, h, positions, eps, r)
        if layer.get("mlp"):
            y = y + feed_forward(W, p + "mlp.", layer["mlp"], h, margins, r)
        x = x + y
        if taps is not None:
            taps.append(x.clone())
    return r(offset_norm(x, W["final.norm"], eps)) @ W["head"].T


def greedy(prompt: List[int], n_new: int, W: Dict[str, torch.Tensor], cfg: dict) -> List[int]:
    """The ``n_new`` tokens greedy decoding appends (the whole sequence runs again per token)."""
    ids, out = list(prompt), []
    for _ in range(n_new):
        nxt = int(forward(ids, W, cfg)[-1].argmax())
        out.append(nxt)
        ids.append(nxt)
    return out
