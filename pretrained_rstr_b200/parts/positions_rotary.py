"""Frequencies of rotary positions: pair i of dims / 2 at position p turns by p * base^(-2 i /
dims); pair i is (i, i + dims / 2) in the rotate-half layout and (2i, 2i + 1) in the interleaved
one.  Kernels compute the angles from these tables and the tokens' positions, or read the
step's table of cosines and sines (:class:`RotaryAngles`)."""
from __future__ import annotations

import hashlib

import torch

from ..csrc import ops


def rotary_frequencies(base: float, dims: int, device, divide_by: float = 1.0,
                       with_lo: bool = False):
    """float32 [max(1, dims / 2)] (a table of one zero when nothing is rotated); ``divide_by``:
    linear scaling of the positions, every frequency divided by it.  ``with_lo``: (hi, lo)
    tables, see :func:`split_frequencies`."""
    if dims < 0 or dims % 2:
        raise ValueError(f"rotary positions need an even number of coordinates, got {dims}")
    half = dims // 2
    freq = [float(base) ** (-2.0 * i / dims) / float(divide_by) for i in range(half)] or [0.0]
    if with_lo:
        return split_frequencies(freq, device)
    return torch.tensor(freq, dtype=torch.float64).to(torch.float32).to(device)


def split_frequencies(freq64, device):
    """(hi, lo) float32 tables of frequencies given in 64-bit: hi is the rounded frequency, lo
    what the rounding left out.  The kernels that take ``freq_lo`` add the two in 64-bit, so the
    angle position x frequency keeps the frequency's full precision."""
    f64 = torch.as_tensor(freq64, dtype=torch.float64)
    hi = f64.to(torch.float32)
    lo = (f64 - hi.to(torch.float64)).to(torch.float32)
    return hi.to(device), lo.to(device)


def yarn_frequencies(base: float, dims: int, factor: float, original: float, fast: float,
                     slow: float, device, with_lo: bool = False):
    """(frequencies float32 [dims / 2], magnitude) of YaRN-scaled rotary positions.  With
    d(t) = dims * ln(original / (2 pi t)) / (2 ln base), lo = max(floor(d(fast)), 0), hi =
    min(ceil(d(slow)), dims - 1) and ramp_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1),
    frequency i is f_i / factor * ramp_i + f_i * (1 - ramp_i) (fast-turning pairs keep their
    frequency, slow ones are interpolated), and cos and sin are both multiplied by the
    magnitude 0.1 * ln(factor) + 1.  ``with_lo``: the frequencies as (hi, lo) tables, see
    :func:`split_frequencies`."""
    import math
    if dims <= 0 or dims % 2:
        raise ValueError(f"rotary positions need an even number of coordinates, got {dims}")

    def d_of(t: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(d_of(fast)), 0)
    hi = min(math.ceil(d_of(slow)), dims - 1)
    freq = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        freq.append(f / factor * ramp + f * (1.0 - ramp))
    table = torch.tensor(freq, dtype=torch.float64).to(torch.float32).to(device)
    if with_lo:
        return split_frequencies(freq, device), 0.1 * math.log(factor) + 1.0
    return table, 0.1 * math.log(factor) + 1.0


def banded_frequencies(base: float, dims: int, factor: float, low: float, high: float,
                       original: float):
    """Frequencies scaled by their wavelength l = 2 pi / f (Llama 3.1's scaling): f where l <
    original / high, f / factor where l > original / low, and between the two the blend (1 - s) f /
    factor + s f with s = (original / l - low) / (high - low).  A list of 64-bit numbers."""
    import math
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        wave = 2.0 * math.pi / f
        if wave < original / high:
            out.append(f)
        elif wave > original / low:
            out.append(f / factor)
        else:
            s = (original / wave - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return out


class RotaryAngles:
    """Cosines and sines of every token's angles, times one ``magnitude``, computed once per step and
    shared by all layers, heads and passes whose frequencies and magnitude are the same."""

    def __init__(self, freq, freq_lo, magnitude: float = 1.0):
        self.freq, self.freq_lo, self.magnitude = freq, freq_lo, float(magnitude)
        mark = hashlib.sha256(freq.cpu().numpy().tobytes() + freq_lo.cpu().numpy().tobytes() +
                              repr(self.magnitude).encode())
        self.key = f"rotary_angles_{mark.hexdigest()[:16]}"

    def table(self, ctx, rows: int):
        """float32 [rows, pairs, 2] of this step."""
        done = ctx.__dict__.setdefault("rotary_done", {})
        out = done.get(self.key)
        if out is None:
            out = ctx.scratch(self.key, (ctx.token_capacity, self.freq.numel(), 2), torch.float32)[:rows]
            ops.rotary_angles(out, ctx.positions, self.freq, self.freq_lo, self.magnitude)
            done[self.key] = out
        return out
