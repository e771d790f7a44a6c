"""Lemunex as data for the engine: tensor names and shapes, random initialisation, named sizes,
registration.  The model is put together by
:func:`pretrained_rstr_b200.models.assembly.build_model` from the parts that
``LemunexConfig.layer_specs()`` names.

Tensor names: ``embed`` and ``head`` [vocab, width], ``embed.norm``, ``final.norm`` [width] and, per
layer i, ``l<i>.norm1`` [width], the mixer's ``l<i>.mix.*`` (``.left.*`` and ``.right.*`` in layers with
two mixers) and the feed-forward's ``l<i>.mlp.*``; matrices are [out, in], biases carry ``.b``.
"""
from __future__ import annotations

import math
from typing import Dict

import torch

from ..config.lemunex import LemunexConfig
from ..config.registry import Architecture, register_architecture
from ..weights.loader import TensorExpectation, normal

#: rows of the decays' low-rank matrix in random models (a file's own tensor says how many it has)
DECAY_RANK = 16


def _mixer_tensors(exp, p: str, entry, d: int, rank) -> None:
    mx = entry["mixer"]
    if entry["type"] == "mamba2":
        h, inner = mx["heads"], mx["heads"] * mx["vdim"]
        channels = inner + 2 * mx["groups"] * mx["state"]
        exp[p + "in"] = TensorExpectation((inner + channels + h, d))
        exp[p + "conv"] = TensorExpectation((channels, mx["conv"]))
        exp[p + "conv.b"] = TensorExpectation((channels,))
        for name in ("dt_bias", "A_log", "D"):
            exp[p + name] = TensorExpectation((h,))
        exp[p + "norm"] = TensorExpectation((inner,))
        exp[p + "o"] = TensorExpectation((d, inner))
        return
    left, right, lp, rp = mx["left"], mx["right"], p + "left.", p + "right."
    h, g = left["heads"], left["kv_heads"]
    for name, rows in (("q", h * left["dim"]), ("k", g * left["dim"]), ("v", g * left["vdim"])):
        exp[lp + name] = TensorExpectation((rows, d))
        exp[lp + name + ".b"] = TensorExpectation((rows,))
    exp[lp + "g"] = TensorExpectation((h, d))
    exp[lp + "o"] = TensorExpectation((d, h * left["vdim"]))
    exp[lp + "o.b"] = TensorExpectation((d,))
    hk, hv = right["heads"] * right["dim"], right["heads"] * right["vdim"]
    for name, rows in (("q", hk), ("k", hk), ("v", hv), ("g", hv)):
        exp[rp + name] = TensorExpectation((rows, d))
    exp[rp + "o"] = TensorExpectation((d, hv))
    exp[rp + "norm"] = TensorExpectation((right["vdim"],))
    free = rank is None
    exp[rp + "a1"] = TensorExpectation((rank or DECAY_RANK, d), free_dims=(0,) if free else ())
    exp[rp + "a2"] = TensorExpectation((hk, rank or DECAY_RANK), free_dims=(1,) if free else ())
    exp[rp + "a2.b"] = TensorExpectation((hk,))


def _gated(exp, p: str, ff: int, d: int) -> None:
    exp[p + "gate"] = TensorExpectation((ff, d))
    exp[p + "up"] = TensorExpectation((ff, d))
    exp[p + "down"] = TensorExpectation((d, ff))


def expected_tensors(cfg: LemunexConfig, rank=None) -> Dict[str, TensorExpectation]:
    """``rank``: rows of the decays' low-rank matrix (None: the file's tensor decides)."""
    d = cfg.width
    exp: Dict[str, TensorExpectation] = {
        "embed": TensorExpectation((cfg.vocab, d)), "embed.norm": TensorExpectation((d,)),
        "final.norm": TensorExpectation((d,)), "head": TensorExpectation((cfg.vocab, d))}
    for i, entry in enumerate(cfg.layers):
        p = f"l{i}."
        exp[p + "norm1"] = TensorExpectation((d,))
        _mixer_tensors(exp, p + "mix.", entry, d, rank)
        mlp = entry.get("mlp")
        if mlp is None:
            continue
        m = p + "mlp."
        if mlp["kind"] == "dense":
            exp[m + "up"] = TensorExpectation((mlp["ff"], d))
            exp[m + "down"] = TensorExpectation((d, mlp["ff"]))
            continue
        router = mlp["router"]
        n = router["experts"] + router.get("identity", 0)
        for e in range(router["experts"]):
            _gated(exp, f"{m}e{e}.", mlp["expert"]["ff"], d)
        exp[m + "router"] = TensorExpectation((n, d))
        exp[m + "correction"] = TensorExpectation((n,))
        if mlp.get("shared"):
            _gated(exp, m + "shared.", mlp["shared"]["ff"], d)
            exp[m + "shared.sg"] = TensorExpectation((1, d))
    return exp


def random_tensors(cfg: LemunexConfig, seed: int) -> Dict[str, torch.Tensor]:
    """Seeded initialisation: matrices N(0, 1/in), the token table N(0, 1), norm weights around their
    neutral value with N(0, 0.1), biases N(0, 0.3) (the decays' N(2, 1)), convolution taps N(0, 0.5),
    D N(1, 0.3), dt_bias N(-2, 1), A_log N(0, 0.7), corrections N(0, 0.05); every tensor from a
    generator of its own."""
    out: Dict[str, torch.Tensor] = {}
    for name, exp in expected_tensors(cfg, rank=DECAY_RANK).items():
        last = name.rsplit(".", 1)[-1]
        std, mean = 1.0 / math.sqrt(exp.shape[-1]), 0.0
        if name == "embed":
            std = 1.0
        elif last == "norm1" or name in ("embed.norm", "final.norm"):
            std = 0.1
        elif last == "norm":
            std, mean = 0.1, 1.0
        elif name.endswith(".a2.b"):
            std, mean = 1.0, 2.0
        elif last == "b":
            std = 0.3
        elif last == "conv":
            std = 0.5
        elif last == "D":
            std, mean = 0.3, 1.0
        elif last == "dt_bias":
            std, mean = 1.0, -2.0
        elif last == "A_log":
            std = 0.7
        elif last == "correction":
            std = 0.05
        out[name] = normal(seed, name, exp.shape, std, mean=mean)
    return out


def _mamba(heads, vdim, state, mlp, groups=1, conv=4, parts=1):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups,
                                        "conv": conv, "norm_groups": parts}, "mlp": mlp}


def _parallel(left, right, mlp, window=512, left_scale=0.8, right_scale=0.6, tau=16.0, base=10000.0,
              rot_dims=None, scaling=(4.0, 256, 32.0, 1.0)):
    heads, kv_heads, dim, vdim = left
    rot = {"base": base, "dims": dim if rot_dims is None else rot_dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                               "scale": 1.0 / math.sqrt(dim), "rot": rot,
                               **({"mask": {"size": window}} if window else {})},
                      "right": dict(zip(("heads", "dim", "vdim"), right), tau=tau),
                      "left_scale": left_scale, "right_scale": right_scale},
            "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, identity, top, ff, shared):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "identity": identity, "top": top},
            "shared": {"ff": shared}}


def _sized(vocab, width, layers, eps=1e-6):
    return {"architecture": "Lemunex", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": layers}


#: Sizes a random-weight model can be asked for by name.  ``lemunex-small`` has the width, head count,
#: vocabulary and number of layers of GPT-2 small: a state-space layer (24 heads of 64 over a state
#: of 128) with a feed-forward of 2,048 and a layer of attention (12 query heads of 64 on 4 key/value
#: heads, window 512) beside gated linear attention (12 heads of 64 x 64), with 8 experts of 512 and 2
#: identity experts of which 3 are chosen and a shared expert of 1,024, take turns.
#: ``lemunex-wide`` has GPT-2 XL's width with heads of 128 (64 in the state-space layers).
NAMED_SIZES = {
    "lemunex-tiny": _sized(300, 72, [
        _parallel((4, 2, 16, 24), (3, 8, 16), _moe(5, 2, 3, 24, 40), window=21, tau=4.0, rot_dims=12),
        _mamba(6, 16, 24, _dense(88), groups=2, conv=3, parts=3),
        _mamba(4, 24, 16, _moe(3, 1, 2, 16, 32)),
        _parallel((2, 1, 24, 16), (2, 24, 8), None, window=40, scaling=None)]),
    "lemunex-small": _sized(50257, 768, [
        (_parallel((12, 4, 64, 64), (12, 64, 64), _moe(8, 2, 3, 512, 1024)) if i % 2
         else _mamba(24, 64, 128, _dense(2048))) for i in range(12)]),
    "lemunex-wide": _sized(50257, 1600, [
        (_parallel((25, 5, 128, 128), (12, 128, 128), _moe(8, 2, 3, 1024, 2048)) if i % 2
         else _mamba(50, 64, 128, _dense(4096))) for i in range(12)]),
}


def build(cfg: LemunexConfig, store, runtime):
    from .assembly import build_model
    return build_model(cfg, store, runtime)


ARCHITECTURE = Architecture(
    name="Lemunex",
    config_class=LemunexConfig,
    build=build,
    expected_tensors=expected_tensors,
    random_tensors=random_tensors,
    named_sizes=NAMED_SIZES,
)
register_architecture(LemunexConfig.identifiers, ARCHITECTURE)
