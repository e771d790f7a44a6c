"""Typed model configurations and the data that describes how layers are arranged.

A configuration class reads the architecture's own ``config.json`` keys once, applies
defaults in one place and validates them (the reference normalises hyper-parameters
the same way: ``src/pretrained/decoder.clj:36-56``).  Everything downstream takes its
sizes and constants from the configuration object; no size lives in code.

Besides sizes, a configuration answers two structural questions as *data*:

``layer_specs()``
    one :class:`LayerSpec` per layer: which mixer, feed-forward, norm and arrangement
    that layer uses, each with its own parameters, so different layers of one model
    may be built from different parts.

``run_order()``
    a list of :class:`RunEntry`: which layer runs when, and whose cache it uses.  A
    layer may appear twice (with the same cache, or with one of its own per run), an entry
    may read another layer's cache, and an entry may have the embedding's output added to the
    stream before it.
"""
from __future__ import annotations

import dataclasses
import json
import os
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional


class ConfigError(ValueError):
    """A config.json that cannot describe a model of the chosen architecture."""


@dataclass(frozen=True)
class PartSpec:
    """Names a registered part (``kind``) and gives its parameters."""

    kind: str
    params: Dict[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class LayerSpec:
    """One layer: its parts, their parameters, and how the block arranges them.

    ``prefix`` is the tensor-name prefix of the layer's weights (``"h.3."``).
    ``arrangement`` names a registered block arrangement (``"pre_norm"``).
    ``norms`` are the layer's norms by the names its arrangement asks for: ``pre_norm``
    wants ``"mixer"`` and ``"feed_forward"``; a block with sandwich norms would name four,
    a parallel block one.  ``width`` is the width of the residual stream.
    ``arrangement_params``: constants and tensor names of the arrangement itself (a scale of
    the stream, gates of the branches); an arrangement that has some is built as
    ``factory(mixer, feed_forward, norms, width, runtime, params=..., store=...)``.
    """

    prefix: str
    arrangement: str
    mixer: PartSpec
    feed_forward: PartSpec
    norms: Dict[str, PartSpec]
    width: int
    arrangement_params: Dict[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class RunEntry:
    """One position in the execution order.

    ``layer``       index into ``layer_specs()`` (weights).
    ``cache_layer`` which cache (pages and state) this entry uses: the index of the layer
                    whose cache it is, or, for a layer that runs several times with a cache
                    of its own each time, any further number (the entry that writes a cache
                    says, by its ``layer``, whose mixer shapes it).
    ``writes_cache`` False when the entry only reads a cache another entry filled.
    ``add_embedding`` the embedding's output (the stream as it was before the first entry)
                    is added to the stream before this entry runs.
    ``join_embedding`` the stream and the embedding's output pass the configuration's
                    ``stream_join_spec()`` before this entry runs.
    """

    layer: int
    cache_layer: int
    writes_cache: bool = True
    add_embedding: bool = False
    join_embedding: bool = False


def looped_run_order(n_layers: int, loop: Optional[Dict[str, int]], first_of_pass) -> List[RunEntry]:
    """Layers 0 .. n_layers - 1 in order, with layers ``start`` .. ``stop`` - 1 of ``loop`` run
    ``times`` times in a row (the same weights; every pass has caches of its own: the first pass
    the layers', further ones numbered after the last layer).  ``first_of_pass(pass number)``
    gives the further fields of a pass's first entry."""
    if loop is None:
        return [RunEntry(i, i) for i in range(n_layers)]
    a, b = loop["start"], loop["stop"]
    order = [RunEntry(i, i) for i in range(a)]
    for rep in range(loop["times"]):
        for i in range(a, b):
            cache = i if rep == 0 else n_layers + (rep - 1) * (b - a) + (i - a)
            order.append(RunEntry(i, cache, True, **(first_of_pass(rep) if i == a else {})))
    return order + [RunEntry(i, i) for i in range(b, n_layers)]



class ModelConfig:
    """Base of all typed configurations."""

    #: HF identifiers this configuration answers to (``architectures[]`` entries and
    #: ``model_type``), used by the registry.
    identifiers: tuple = ()

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "ModelConfig":
        raise NotImplementedError

    def to_dict(self) -> Dict[str, Any]:
        raise NotImplementedError

    # --- structure as data -------------------------------------------------
    def layer_specs(self) -> List[LayerSpec]:
        raise NotImplementedError

    def run_order(self) -> List[RunEntry]:
        return [RunEntry(i, i, True) for i in range(len(self.layer_specs()))]

    def embedding_spec(self) -> PartSpec:
        raise NotImplementedError

    def position_spec(self) -> PartSpec:
        return PartSpec("none")

    def stream_join_spec(self) -> Optional[PartSpec]:
        """How entries with ``join_embedding`` join the stream with the embedding's output."""
        return None

    def final_norm_spec(self) -> PartSpec:
        raise NotImplementedError

    def head_spec(self) -> PartSpec:
        raise NotImplementedError

    @property
    def max_positions(self) -> int:
        raise NotImplementedError

    # --- helpers -------------------------------------------------------------
    @classmethod
    def from_folder(cls, folder: str) -> "ModelConfig":
        with open(os.path.join(folder, "config.json"), "r", encoding="utf-8") as fh:
            return cls.from_dict(json.load(fh))

    def save(self, folder: str) -> None:
        os.makedirs(folder, exist_ok=True)
        with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as fh:
            json.dump(self.to_dict(), fh, indent=2, sort_keys=True)
            fh.write("\n")


def _require_int(raw: Dict[str, Any], key: str, default: Optional[int] = None,
                 minimum: int = 1) -> int:
    value = raw.get(key, default)
    if value is None:
        raise ConfigError(f"config.json: missing required key '{key}'")
    if isinstance(value, bool) or not isinstance(value, int):
        raise ConfigError(f"config.json: '{key}' must be an integer, got {value!r}")
    if value < minimum:
        raise ConfigError(f"config.json: '{key}' must be >= {minimum}, got {value}")
    return value


def _require_float(raw: Dict[str, Any], key: str, default: float) -> float:
    value = raw.get(key, default)
    if isinstance(value, bool) or not isinstance(value, (int, float)):
        raise ConfigError(f"config.json: '{key}' must be a number, got {value!r}")
    return float(value)


def _require_bool(raw: Dict[str, Any], key: str, default: bool) -> bool:
    value = raw.get(key, default)
    if not isinstance(value, bool):
        raise ConfigError(f"config.json: '{key}' must be true or false, got {value!r}")
    return value


def config_int(d, key: str, where: str, minimum: int = 1) -> int:
    """``d[key]``, an integer that is at least ``minimum``; ``where`` names ``d`` in the error."""
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, int) or v < minimum:
        raise ConfigError(f"config.json: {where}.{key} must be an integer >= {minimum}, got {v!r}")
    return v


def config_number(d, key: str, where: str) -> float:
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: {where}.{key} must be a number, got {v!r}")
    return float(v)


def replace(config, **changes):
    """``dataclasses.replace`` that re-validates."""
    return type(config).from_dict({**config.to_dict(), **changes})


__all__ = ["ConfigError", "PartSpec", "LayerSpec", "RunEntry", "ModelConfig", "looped_run_order",
           "config_int", "config_number", "replace", "dataclasses"]
