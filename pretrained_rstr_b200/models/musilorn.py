"""Musilorn as data for the engine: tensor names and shapes, random initialisation, named
sizes, registration.  The model is put together by
:func:`pretrained_rstr_b200.models.assembly.build_model` from the parts that
``MusilornConfig.layer_specs()`` names, in the order ``run_order()`` gives.

Tensor names: ``embed`` and ``head`` [vocab, width], ``final.norm`` [width], ``loop.in`` [width,
2 width] (with a loop) and per layer i ``l<i>.norm1``, ``l<i>.norm1b``, with a feed-forward
``l<i>.norm2``, ``l<i>.norm2b`` [width], the mixer's ``l<i>.mix.*`` and the feed-forward's
``l<i>.mlp.*``; matrices are [out, in], convolutions [channels, taps]; every norm over the stream
has a bias, its name with ``.b`` added.
"""
from __future__ import annotations

import math
from typing import Dict

import torch

from ..config.musilorn import MusilornConfig
from ..config.registry import Architecture, register_architecture
from ..weights.loader import TensorExpectation, normal


def expected_tensors(cfg: MusilornConfig) -> Dict[str, TensorExpectation]:
    d = cfg.width
    exp: Dict[str, TensorExpectation] = {}

    def add(name, *shape):
        exp[name] = TensorExpectation(tuple(shape))

    def norm(name):
        add(name, d)
        add(name + ".b", d)

    add("embed", cfg.vocab, d)
    add("head", cfg.vocab, d)
    norm("final.norm")
    if cfg.loop is not None:
        add("loop.in", d, 2 * d)
    for i, entry in enumerate(cfg.layers):
        p, mx, mlp = f"l{i}.", entry["mixer"], entry.get("mlp")
        m = p + "mix."
        h, dim, vd = mx["heads"], mx["dim"], mx["vdim"]
        norm(p + "norm1")
        norm(p + "norm1b")
        if entry["type"] == "attention":
            for s, n in (("q", h), ("k", mx["kv_heads"])):
                add(m + s, n * dim, d)
                add(m + s + ".norm", dim)
                add(m + s + ".conv", n * dim, mx["conv"])
        else:
            add(m + "q", h * dim, d)
            add(m + "k", h * dim, d)
            add(m + "v", h * vd, d)
            add(m + "g", h * vd, d)
        add(m + "o", d, h * vd)
        if mlp is None:
            continue
        norm(p + "norm2")
        norm(p + "norm2b")
        add(p + "mlp.gate", mlp["ff"], d)
        add(p + "mlp.up", mlp["ff"], d)
        add(p + "mlp.down", d, mlp["ff"])
    return exp


def random_tensors(cfg: MusilornConfig, seed: int) -> Dict[str, torch.Tensor]:
    """Seeded initialisation: matrices N(0, 1/in), the token table N(0, 1), norm weights 1 +
    N(0, 0.1), their biases N(0, 0.1), convolution taps N(0, 0.5); every tensor from a generator of
    its own."""
    out: Dict[str, torch.Tensor] = {}
    for name, exp in expected_tensors(cfg).items():
        if name == "embed":
            out[name] = normal(seed, name, exp.shape, 1.0)
        elif name.endswith(".b"):
            out[name] = normal(seed, name, exp.shape, 0.1)
        elif len(exp.shape) == 1:
            out[name] = normal(seed, name, exp.shape, 0.1, mean=1.0)
        elif name.endswith(".conv"):
            out[name] = normal(seed, name, exp.shape, 0.5)
        else:
            out[name] = normal(seed, name, exp.shape, 1.0 / math.sqrt(exp.shape[-1]))
    return out


def _attention(heads, kv_heads, dim, ff, conv=4, rot_dims=None, base=500000.0, softcap=30.0,
               scaling=(4.0, 1.0, 4.0, 512)):
    rot = {"base": base, "dims": dim if rot_dims is None else rot_dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv,
                      "scale": 1.0 / math.sqrt(dim), "softcap": softcap, "rot": rot},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _retention(heads, dim, vdim, ff, rot_dims=None, base=10000.0):
    # decays 1 - 2^-(5 + j): short memories on the first heads, long ones on the last
    return {"type": "retention",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim,
                      "decay": [1.0 - 2.0 ** (-5.0 - 3.0 * j / max(1, heads - 1)) for j in range(heads)],
                      "rot": {"base": base, "dims": dim if rot_dims is None else rot_dims}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _sized(vocab, width, layers, loop=None, mult=0.5, cap=30.0, eps=1e-5):
    out = {"architecture": "Musilorn", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "residual_mult": mult, "logit_softcap": cap, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


#: Sizes a random-weight model can be asked for by name.  ``musilorn-small`` has the width, head
#: count, vocabulary and number of layer runs of GPT-2 small (8 layers of which 2 run three times:
#: 12 runs): an attention layer (12 query heads of 64 on 4 key/value heads, 4 taps) and a retention
#: layer (12 heads of 64 x 64) take turns, every layer with a gated feed-forward of 2,048.
#: ``musilorn-wide`` has GPT-2 XL's width with heads of 128.
NAMED_SIZES = {
    "musilorn-tiny": _sized(300, 72, [
        _retention(3, 16, 24, 56, rot_dims=8),
        _attention(4, 2, 24, None, conv=2, rot_dims=16, softcap=8.0, scaling=None),
        _attention(2, 1, 16, 88, conv=5, softcap=12.0, scaling=(3.0, 1.0, 2.5, 96)),
        _retention(2, 24, 8, None)], loop=(1, 3, 2), mult=0.6, cap=9.0),
    "musilorn-small": _sized(50257, 768, [
        (_retention(12, 64, 64, 2048) if i % 2 else _attention(12, 4, 64, 2048))
        for i in range(8)], loop=(2, 4, 3)),
    "musilorn-wide": _sized(50257, 1600, [
        (_retention(25, 128, 128, 4096) if i % 2 else _attention(25, 5, 128, 4096))
        for i in range(8)], loop=(2, 4, 3)),
}


def build(cfg: MusilornConfig, store, runtime):
    from .assembly import build_model
    return build_model(cfg, store, runtime)


ARCHITECTURE = Architecture(
    name="Musilorn",
    config_class=MusilornConfig,
    build=build,
    expected_tensors=expected_tensors,
    random_tensors=random_tensors,
    named_sizes=NAMED_SIZES,
)
register_architecture(MusilornConfig.identifiers, ARCHITECTURE)
