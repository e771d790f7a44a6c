"""Lemunex configuration: a decoder whose layers are listed one by one in ``config.json``.

Keys read (nothing else exists in the design):

``vocab``, ``width``   sizes of the token table, of the head (a matrix of its own) and of the stream
``norm.eps``           epsilon of every root-mean-square norm
``layers[i]``          ``type`` (``parallel`` or ``mamba2``), ``mixer`` (the mixer's sizes and
                       constants) and ``mlp``: ``kind`` dense with ``ff``; or ``kind`` moe with
                       ``expert.ff``, ``router`` (``experts``, ``identity``, ``top``) and optionally
                       ``shared.ff``; or null for a layer without a feed-forward

The embedding's output is normed before the first layer.  A layer has ONE norm, and its mixer and its
feed-forward both read it: x <- x + (mixer(h) + feed_forward(h)).  These norms' weights are stored
around zero (1 + w).  ``mamba2`` layers have a state-space mixer (``heads``, ``vdim``, ``state``,
``groups``, ``conv``, ``norm_groups``).  ``parallel`` layers have two mixers side by side, ``mixer.left``
(softmax attention with grouped key/value heads, biases on all four projections, a sliding window
``mask.size``, interleaved rotary pairs with YaRN-scaled frequencies and a gate per head) and
``mixer.right`` (gated linear attention: ``heads``, ``dim``, ``vdim``, ``tau``), summed with
``left_scale`` and ``right_scale``.  The dense feed-forward squares a relu; the other routes a token
to ``top`` of ``experts + identity`` experts (the last ``identity`` give back their input) by softmax
scores with a correction for the choice, beside a shared expert with a gate of its own.

The design names no position limit; a loaded model's limit is what its page pool holds
(``position_limit`` caps it).
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List

from .base import (ConfigError, LayerSpec, ModelConfig, PartSpec,
                   config_int as _int, config_number as _num)

_TYPES = ("parallel", "mamba2")
#: the constant the design fixes: norms of the stream multiply by 1 + w
NORM_OFFSET = 1.0


def _check_rot(rot, most: int, where: str) -> None:
    dims = _int(rot, "dims", where, 0)
    if _num(rot, "base", where) <= 0.0:
        raise ConfigError(f"config.json: {where}.base must be positive")
    if dims % 2 or dims > most:
        raise ConfigError(f"config.json: {where}.dims must be even and at most {most}, got {dims}")
    sc = rot.get("scaling")
    if sc is None:
        return
    for key in ("factor", "original", "fast", "slow"):
        if _num(sc, key, where + ".scaling") <= 0.0:
            raise ConfigError(f"config.json: {where}.scaling.{key} must be positive")


def _check_parallel(mx, where: str) -> None:
    left, right = mx.get("left"), mx.get("right")
    for key in ("heads", "kv_heads", "dim", "vdim"):
        _int(left, key, where + ".left")
    if left["heads"] % left["kv_heads"]:
        raise ConfigError(f"config.json: {where}.left.heads is no multiple of kv_heads")
    _num(left, "scale", where + ".left")
    if left.get("rot") is not None:
        _check_rot(left["rot"], left["dim"], where + ".left.rot")
    if left.get("mask") is not None:
        _int(left["mask"], "size", where + ".left.mask")
    for key in ("heads", "dim", "vdim"):
        _int(right, key, where + ".right")
    if _num(right, "tau", where + ".right") <= 0.0:
        raise ConfigError(f"config.json: {where}.right.tau must be positive")
    _num(mx, "left_scale", where)
    _num(mx, "right_scale", where)


def _check_mamba2(mx, where: str) -> None:
    for key in ("heads", "vdim", "state", "groups", "conv", "norm_groups"):
        _int(mx, key, where)
    if mx["heads"] % mx["groups"]:
        raise ConfigError(f"config.json: {where}.heads is no multiple of groups")
    if mx["heads"] * mx["vdim"] % mx["norm_groups"]:
        raise ConfigError(f"config.json: {where}: heads * vdim does not split into norm_groups parts")


def _check_mlp(mlp, where: str) -> None:
    kind = mlp.get("kind") if isinstance(mlp, dict) else None
    if kind == "dense":
        _int(mlp, "ff", where)
        return
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind must be 'dense' or 'moe' (or mlp null)")
    _int(mlp.get("expert"), "ff", where + ".expert")
    router = mlp.get("router")
    experts, top = _int(router, "experts", where + ".router"), _int(router, "top", where + ".router")
    identity = _int(router, "identity", where + ".router", 0) if "identity" in router else 0
    if top > experts + identity:
        raise ConfigError(f"config.json: {where}.router.top is {top} of {experts + identity} experts")
    if mlp.get("shared") is not None:
        _int(mlp["shared"], "ff", where + ".shared")


@dataclass(frozen=True)
class LemunexConfig(ModelConfig):
    vocab: int
    width: int
    eps: float
    layers: tuple                           # the raw layer entries, validated
    position_limit: int = 1 << 20
    raw: Dict[str, Any] = field(default_factory=dict, compare=False, repr=False)

    identifiers = ("Lemunex",)

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "LemunexConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        cfg = cls(vocab=_int(raw, "vocab", "config"), width=_int(raw, "width", "config"),
                  eps=_num(raw.get("norm"), "eps", "norm"), layers=tuple(copy.deepcopy(layers)),
                  position_limit=int(raw.get("position_limit", 1 << 20)), raw=copy.deepcopy(raw))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.eps < 0.0:
            raise ConfigError("config.json: norm.eps must not be negative")
        for i, entry in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(entry, dict) or entry.get("type") not in _TYPES:
                raise ConfigError(f"config.json: {where}.type must be one of {list(_TYPES)}")
            mx = entry.get("mixer")
            if not isinstance(mx, dict):
                raise ConfigError(f"config.json: {where}.mixer must be an object")
            (_check_mamba2 if entry["type"] == "mamba2" else _check_parallel)(mx, where + ".mixer")
            if entry.get("mlp") is not None:
                _check_mlp(entry["mlp"], where + ".mlp")

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": "Lemunex", "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.eps}, "layers": copy.deepcopy(list(self.layers))}
        if self.position_limit != 1 << 20:
            out["position_limit"] = self.position_limit
        return out

    # ---------------------------------------------------------------- structure
    def _mixer_spec(self, entry, p: str) -> PartSpec:
        mx = entry["mixer"]
        if entry["type"] == "mamba2":
            names = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias",
                     "A_log": "A_log", "D": "D", "norm": "norm", "out": "o"}
            return PartSpec("state_space", {
                "width": self.width, "heads": mx["heads"], "vdim": mx["vdim"], "state": mx["state"],
                "groups": mx["groups"], "taps": mx["conv"], "norm_parts": mx["norm_groups"],
                "eps": self.eps, "weights": {k: p + v for k, v in names.items()}})
        left, right = mx["left"], mx["right"]
        rot = left.get("rot") or {}
        lw = {"q": "q", "k": "k", "v": "v", "gate": "g", "out": "o", "q_bias": "q.b", "k_bias": "k.b",
              "v_bias": "v.b", "out_bias": "o.b"}
        rw = {"q": "q", "k": "k", "v": "v", "gate": "g", "out": "o", "norm": "norm", "decay_down": "a1",
              "decay_up": "a2", "decay_bias": "a2.b"}
        return PartSpec("side_by_side", {
            "left": PartSpec("window_attention", {
                "width": self.width, "heads": left["heads"], "kv_heads": left["kv_heads"],
                "dim": left["dim"], "vdim": left["vdim"], "scale": float(left["scale"]),
                "eps": self.eps, "window": (left.get("mask") or {}).get("size"),
                "rot_dims": rot.get("dims", 0), "rot_base": float(rot.get("base", 10000.0)),
                "rot_layout": "interleaved", "rot_yarn": copy.deepcopy(rot.get("scaling")),
                "bias": True, "out_bias": True, "head_gate": True,
                "weights": {k: p + "left." + v for k, v in lw.items()}}),
            "right": PartSpec("gated_linear_attention", {
                "width": self.width, "heads": right["heads"], "dim": right["dim"],
                "vdim": right["vdim"], "tau": float(right["tau"]), "eps": self.eps,
                "weights": {k: p + "right." + v for k, v in rw.items()}}),
            "left_scale": float(mx["left_scale"]), "right_scale": float(mx["right_scale"])})

    def _ff_spec(self, mlp, p: str) -> PartSpec:
        if mlp is None:
            return PartSpec("none", {})
        if mlp["kind"] == "dense":
            return PartSpec("act_mlp", {"width": self.width, "inner": mlp["ff"],
                                        "activation": "relu_squared",
                                        "weights": {"up": p + "up", "down": p + "down"}})
        router, shared = mlp["router"], mlp.get("shared") or {}
        return PartSpec("gated_moe", {
            "width": self.width, "experts": router["experts"], "top": router["top"],
            "identity": router.get("identity", 0), "inner": mlp["expert"]["ff"],
            "shared_inner": shared.get("ff", 0), "shared_gate": True, "correction": True,
            "limit": 0.0, "act_alpha": 1.0, "up_shift": 0.0, "score": "softmax",
            "renormalize": False, "router_bias": False, "prefix": p})

    def _norm_spec(self, name: str) -> PartSpec:
        return PartSpec("rms_norm", {"weight": name, "eps": self.eps, "size": self.width,
                                     "offset": NORM_OFFSET})

    def layer_specs(self) -> List[LayerSpec]:
        specs = []
        for i, entry in enumerate(self.layers):
            p = f"l{i}."
            specs.append(LayerSpec(prefix=p, arrangement="parallel",
                                   mixer=self._mixer_spec(entry, p + "mix."),
                                   feed_forward=self._ff_spec(entry.get("mlp"), p + "mlp."),
                                   norms={"shared": self._norm_spec(p + "norm1")}, width=self.width))
        return specs

    def embedding_spec(self) -> PartSpec:
        return PartSpec("normed_token_embedding", {
            "weights": "embed", "norm": "embed.norm", "vocab": self.vocab, "width": self.width,
            "eps": self.eps, "offset": NORM_OFFSET})

    def final_norm_spec(self) -> PartSpec:
        return self._norm_spec("final.norm")

    def head_spec(self) -> PartSpec:
        return PartSpec("linear_head", {"weights": "head", "vocab": self.vocab, "width": self.width})

    @property
    def max_positions(self) -> int:
        return self.position_limit
