"""Typed configuration of the Zepilorn decoder.

``config.json`` of this design is nested: ``layers`` is a list with one entry per layer, each naming its mixer
(``type``: ``attention``, ``latent_attention`` or ``lightning``), the mixer's sizes and constants (``mixer``) and its
feed-forward (``mlp``: ``kind`` ``dense`` with ``ff``, or null for none).  An attention layer may name an earlier
attention layer whose keys and values it reads (``mixer.kv_from``).  Model-wide: ``vocab``, ``width``, ``norm.eps``.
Every size and constant is read from here (or from a tensor's shape); the class checks what each kind needs and keeps
the layer entries as they were written, so that ``to_dict`` gives the file back.
"""
from __future__ import annotations

import copy
import math
from dataclasses import dataclass, field
from typing import Any

from .base import ConfigError, as_float, as_int

SIZE_KEYS = {"attention": ("heads", "kv_heads", "dim", "vdim"),
             "latent_attention": ("heads", "dim", "vdim", "kv_rank"),
             "lightning": ("heads", "dim", "vdim")}
SCALING_KEYS = ("factor", "original", "fast", "slow")


def _section(raw: dict, key: str, where: str = "config.json") -> dict:
    v = raw.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where} lacks the section {key!r}")
    return v


def _positive(v: Any, key: str) -> float:
    x = as_float(v, key)
    if not x > 0:
        raise ConfigError(f"{key} must be positive, got {x}")
    return x


def _mask(section: dict, where: str) -> None:
    mask = section.get("mask")
    if mask is None:
        return
    if not isinstance(mask, dict):
        raise ConfigError(f"{where}.mask must be a section")
    as_int(mask.get("size"), f"{where}.mask.size", minimum=1)


def _rotation(section: dict, where: str, most: int) -> None:
    rot = section.get("rot")
    if rot is None:
        return
    if not isinstance(rot, dict):
        raise ConfigError(f"{where}.rot must be a section")
    base = _positive(rot.get("base"), f"{where}.rot.base")
    dims = as_int(rot.get("dims", most), f"{where}.rot.dims", minimum=0)
    if dims % 2 or dims > most:
        raise ConfigError(f"{where}.rot.dims must be even and at most {most}, got {dims}")
    sc = rot.get("scaling")
    if sc is None:
        return
    if not isinstance(sc, dict):
        raise ConfigError(f"{where}.rot.scaling must be a section")
    for key in SCALING_KEYS:
        _positive(sc.get(key), f"{where}.rot.scaling.{key}")
    if math.log(base) == 0.0:
        raise ConfigError(f"{where}.rot.base must not be 1 when the rotation is scaled")


def rotated_dims(mixer: dict) -> int:
    """How many entries of a head are rotated (0: none)."""
    rot = mixer.get("rot")
    return int(rot.get("dims", mixer["dim"])) if rot else 0


@dataclass
class ZepilornConfig:
    vocab: int
    width: int
    layers: list[dict[str, Any]]
    norm_eps: float = 1e-6
    max_positions: int = 32768               # the design has no table of positions; this is the context an engine is
                                             # made for when its caller names none (the key `max_positions` overrides it)
    eos_token_ids: list[int] = field(default_factory=list)

    architecture = "Zepilorn"
    model_type = "zepilorn"

    # what the engine and the command line ask of any config
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def max_position_embeddings(self) -> int:
        return self.max_positions

    @classmethod
    def from_dict(cls, raw: dict) -> "ZepilornConfig":
        if not isinstance(raw.get("layers"), list) or not raw["layers"]:
            raise ConfigError("config.json lacks 'layers' (a list with one entry per layer)")
        for key in ("vocab", "width"):
            if key not in raw:
                raise ConfigError(f"config.json lacks required key {key!r}")
        cfg = cls(vocab=as_int(raw["vocab"], "vocab", minimum=1), width=as_int(raw["width"], "width", minimum=1),
                  layers=copy.deepcopy(raw["layers"]),
                  norm_eps=as_float(_section(raw, "norm").get("eps", 1e-6), "norm.eps"),
                  max_positions=as_int(raw.get("max_positions", 32768), "max_positions", minimum=1))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = layer.get("type") if isinstance(layer, dict) else layer
            if kind not in SIZE_KEYS:
                raise ConfigError(f"{where}: 'type' must be one of {list(SIZE_KEYS)}, got {kind!r}")
            m = _section(layer, "mixer", where)
            w = where + ".mixer"
            for key in SIZE_KEYS[kind]:
                as_int(m.get(key), f"{w}.{key}", minimum=1)
            if kind == "lightning":
                decay = m.get("decay")
                if not isinstance(decay, list) or len(decay) != m["heads"]:
                    raise ConfigError(f"{w}.decay must be a list with one number per head ({m['heads']})")
                for h, v in enumerate(decay):
                    as_float(v, f"{w}.decay[{h}]")
            else:
                as_float(m.get("scale"), f"{w}.scale")
                _mask(m, w)
            if kind == "attention":
                if m["heads"] % m["kv_heads"]:
                    raise ConfigError(f"{w}: heads must be a multiple of kv_heads")
                _rotation(m, w, m["dim"])
                if m.get("kv_from") is not None:
                    self._check_source(i, m, w)
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                raise ConfigError(f"{where}: 'mlp' must be null or of kind 'dense'")
            as_int(mlp.get("ff"), f"{where}.mlp.ff", minimum=1)

    def _check_source(self, i: int, m: dict, w: str) -> None:
        j = as_int(m["kv_from"], f"{w}.kv_from", minimum=0)
        src = self.layers[j] if j < i else None
        if src is None or src.get("type") != "attention" or src["mixer"].get("kv_from") is not None:
            raise ConfigError(f"{w}.kv_from must name an earlier attention layer with projections of its own, got {j}")
        for key in ("kv_heads", "dim", "vdim"):
            if src["mixer"][key] != m[key]:
                raise ConfigError(f"{w}.kv_from: {key} is {m[key]}, layer {j} has {src['mixer'][key]}")

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(self.layers)}
        if self.max_positions != 32768:
            out["max_positions"] = self.max_positions
        return out
