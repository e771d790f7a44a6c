"""Musilorn configuration: a decoder whose layers are listed one by one in ``config.json``, some
of which may run several times in a row.

Keys read (nothing else exists in the design):

``vocab``, ``width``       sizes of the token table / head and of the residual stream
``norm.eps``               epsilon of every norm
``residual_mult``          constant on what a branch adds to the stream
``logit_softcap``          logits are cap * tanh(logits / cap)
``layers[i]``              ``type`` (the mixer: ``attention`` or ``retention``), ``mixer`` (its sizes
                           and constants) and ``mlp`` (``kind`` dense with ``ff``, or null for a
                           layer without a feed-forward)
``loop``                   optional ``start``, ``stop``, ``times``: layers start .. stop - 1 run
                           ``times`` times in a row with the same weights, every pass with a cache
                           and state of its own; before every pass, the first too, the stream
                           becomes W [stream; embedding's output] (tensor ``loop.in``)

A layer norms each branch before and after: x <- x + m norm1b(mixer(norm1(x))), x <- x + m
norm2b(mlp(norm2(x))), all of them layer norms with weight and bias.  ``attention``: grouped
query heads, a short causal convolution on queries and keys, the convolved keys as values, a
norm per head before a rotation of interleaved pairs (frequencies optionally scaled by
wavelength), a cap on scores, causal softmax whose denominator has 1 added.  ``retention``: linear
attention with a fixed decay per head, unit norm per head and a SiLU gate.  The feed-forward is
gated by the tanh form of gelu.

The design names no position limit; a loaded model's limit is what its page pool holds
(``position_limit`` caps it).
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .base import (ConfigError, LayerSpec, ModelConfig, PartSpec, RunEntry, config_int as _int,
                   config_number as _num, looped_run_order)

_MIXERS = ("attention", "retention")
#: constants the design fixes
SINK_SCORE = 0.0            # the softmax's denominator has exp(0) = 1 added


def _positive(d, key: str, where: str) -> float:
    v = _num(d, key, where)
    if v <= 0.0:
        raise ConfigError(f"config.json: {where}.{key} must be positive, got {v!r}")
    return v


def _check_rot(rot, most: int, where: str) -> None:
    dims = _int(rot, "dims", where, 0)
    _positive(rot, "base", where)
    if dims % 2 or dims > most:
        raise ConfigError(f"config.json: {where}.dims must be even and at most {most}, got {dims}")
    sc = rot.get("scaling")
    if sc is not None:
        for key in ("factor", "low", "high", "original"):
            _positive(sc, key, where + ".scaling")


@dataclass(frozen=True)
class MusilornConfig(ModelConfig):
    vocab: int
    width: int
    eps: float
    residual_mult: float
    logit_softcap: Optional[float]
    layers: tuple                           # the raw layer entries, validated
    loop: Optional[Dict[str, int]] = None
    position_limit: int = 1 << 20
    raw: Dict[str, Any] = field(default_factory=dict, compare=False, repr=False)

    identifiers = ("Musilorn",)

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "MusilornConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        loop = raw.get("loop")
        if loop is not None:
            loop = {"start": _int(loop, "start", "loop", 0), "stop": _int(loop, "stop", "loop", 0),
                    "times": _int(loop, "times", "loop", 1)}
        cap = raw.get("logit_softcap")
        cfg = cls(vocab=_int(raw, "vocab", "config"), width=_int(raw, "width", "config"),
                  eps=_num(raw.get("norm"), "eps", "norm"),
                  residual_mult=_num(raw, "residual_mult", "config"),
                  logit_softcap=None if cap is None else _positive(raw, "logit_softcap", "config"),
                  layers=tuple(copy.deepcopy(layers)), loop=loop,
                  position_limit=int(raw.get("position_limit", 1 << 20)), raw=copy.deepcopy(raw))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.eps < 0.0:
            raise ConfigError("config.json: norm.eps must not be negative")
        if self.loop is not None and not 0 <= self.loop["start"] <= self.loop["stop"] <= len(self.layers):
            raise ConfigError(f"config.json: loop {self.loop} does not lie within the "
                              f"{len(self.layers)} layers")
        for i, entry in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(entry, dict) or entry.get("type") not in _MIXERS:
                raise ConfigError(f"config.json: {where}.type must be one of {list(_MIXERS)}")
            mx = entry.get("mixer")
            if not isinstance(mx, dict):
                raise ConfigError(f"config.json: {where}.mixer must be an object")
            where += ".mixer"
            for key in ("heads", "dim", "vdim"):
                _int(mx, key, where)
            _check_rot(mx.get("rot"), mx["dim"], where + ".rot")
            if entry["type"] == "attention":
                if mx["heads"] % _int(mx, "kv_heads", where):
                    raise ConfigError(f"config.json: {where}.heads is no multiple of kv_heads")
                if mx["vdim"] != mx["dim"]:
                    raise ConfigError(f"config.json: {where}: keys are the values, so vdim must equal "
                                      f"dim, got {mx['vdim']} and {mx['dim']}")
                _int(mx, "conv", where)
                _num(mx, "scale", where)
                if mx.get("softcap") is not None:
                    _positive(mx, "softcap", where)
            else:
                if mx["rot"].get("scaling") is not None:
                    raise ConfigError(f"config.json: {where}.rot.scaling: retention's frequencies have "
                                      f"no scaling")
                decay = mx.get("decay")
                if not isinstance(decay, list) or len(decay) != mx["heads"] or \
                        any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
                    raise ConfigError(f"config.json: {where}.decay must list one number per head")
            mlp = entry.get("mlp")
            if mlp is None:
                continue
            if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                raise ConfigError(f"config.json: layers[{i}].mlp.kind must be 'dense' (or mlp null)")
            _int(mlp, "ff", f"layers[{i}].mlp")

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {
            "architecture": "Musilorn", "vocab": self.vocab, "width": self.width,
            "norm": {"eps": self.eps}, "residual_mult": self.residual_mult,
            "layers": copy.deepcopy(list(self.layers))}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        if self.loop is not None:
            out["loop"] = dict(self.loop)
        if self.position_limit != 1 << 20:
            out["position_limit"] = self.position_limit
        return out

    # ---------------------------------------------------------------- structure
    def _mixer_spec(self, entry, p: str) -> PartSpec:
        mx, rot, m = entry["mixer"], entry["mixer"]["rot"], p + "mix."
        common = {"width": self.width, "heads": mx["heads"], "dim": mx["dim"], "vdim": mx["vdim"],
                  "eps": self.eps, "rot_base": float(rot["base"]), "rot_dims": rot["dims"]}
        if entry["type"] == "retention":
            return PartSpec("retention", {
                **common, "decay": [float(d) for d in mx["decay"]],
                "k_scale": float(mx["dim"]) ** -0.5,
                "weights": {"q": m + "q", "k": m + "k", "v": m + "v", "gate": m + "g", "out": m + "o"}})
        return PartSpec("window_attention", {
            **common, "kv_heads": mx["kv_heads"], "scale": float(mx["scale"]),
            "softcap": mx.get("softcap"), "conv": mx["conv"], "keys_are_values": True,
            "qk_norm": "head", "rot_layout": "interleaved",
            "rot_bands": copy.deepcopy(rot.get("scaling")), "sink_score": SINK_SCORE,
            "weights": {"q": m + "q", "k": m + "k", "q_conv": m + "q.conv", "k_conv": m + "k.conv",
                        "q_norm": m + "q.norm", "k_norm": m + "k.norm", "out": m + "o"}})

    def _norm_spec(self, name: str) -> PartSpec:
        return PartSpec("layer_norm", {"weight": name, "bias": name + ".b", "eps": self.eps,
                                       "size": self.width})

    def layer_specs(self) -> List[LayerSpec]:
        specs = []
        for i, entry in enumerate(self.layers):
            p, mlp = f"l{i}.", entry.get("mlp")
            norms = {"mixer": self._norm_spec(p + "norm1"), "mixer_after": self._norm_spec(p + "norm1b")}
            if mlp is None:
                ff = PartSpec("none", {})
            else:
                norms["feed_forward"] = self._norm_spec(p + "norm2")
                norms["feed_forward_after"] = self._norm_spec(p + "norm2b")
                ff = PartSpec("gated_mlp", {
                    "width": self.width, "inner": mlp["ff"], "activation": "gelu_tanh",
                    "weights": {"gate": p + "mlp.gate", "up": p + "mlp.up", "down": p + "mlp.down"}})
            specs.append(LayerSpec(prefix=p, arrangement="sandwich", mixer=self._mixer_spec(entry, p),
                                   feed_forward=ff, norms=norms, width=self.width,
                                   arrangement_params={"residual_mult": self.residual_mult}))
        return specs

    def run_order(self) -> List[RunEntry]:
        return looped_run_order(len(self.layers), self.loop, lambda rep: {"join_embedding": True})

    def embedding_spec(self) -> PartSpec:
        return PartSpec("scaled_token_embedding", {"weights": "embed", "vocab": self.vocab,
                                                   "width": self.width, "scale": 1.0})

    def stream_join_spec(self) -> Optional[PartSpec]:
        if self.loop is None:
            return None
        return PartSpec("linear_join", {"weights": "loop.in", "width": self.width})

    def final_norm_spec(self) -> PartSpec:
        return self._norm_spec("final.norm")

    def head_spec(self) -> PartSpec:
        return PartSpec("linear_head", {"weights": "head", "vocab": self.vocab, "width": self.width,
                                        "softcap": self.logit_softcap})

    @property
    def max_positions(self) -> int:
        return self.position_limit
