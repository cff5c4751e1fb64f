"""Typed configuration of the Gakenex decoder.

``config.json`` of this design is nested: ``layers`` is a list with one entry per layer, each naming its mixer (``type``:
``attention``), the mixer's sizes and constants (``mixer``) and its feed-forward (``mlp``: ``kind`` ``dense`` with ``ff``
and ``limit``, ``kind`` ``moe`` with ``router.experts``, ``router.top`` and ``expert.ff``, or null for none).  Model-wide:
``vocab``, ``width``, ``norm.eps``, ``max_positions`` (rows of the table of positions) and ``logit_softcap``.  Every size
and constant is read from here; the class checks what each kind needs and keeps the layer entries as they were written,
so that ``to_dict`` gives the file back.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any

from .base import ConfigError, as_float, as_int

SIZE_KEYS = ("heads", "kv_heads", "dim", "vdim")


def _section(raw: dict, key: str, where: str = "config.json") -> dict:
    v = raw.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where} lacks the section {key!r}")
    return v


@dataclass
class GakenexConfig:
    vocab: int
    width: int
    layers: list[dict[str, Any]]
    max_positions: int
    norm_eps: float = 1e-6
    logit_softcap: float = 0.0               # 0: the logits are left as they are
    eos_token_ids: list[int] = field(default_factory=list)

    architecture = "Gakenex"
    model_type = "gakenex"

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
    def from_dict(cls, raw: dict) -> "GakenexConfig":
        if not isinstance(raw.get("layers"), list) or not raw["layers"]:
            raise ConfigError("config.json lacks 'layers' (a list with one entry per layer)")
        for key in ("vocab", "width", "max_positions"):
            if key not in raw:
                raise ConfigError(f"config.json lacks required key {key!r}")
        cap = raw.get("logit_softcap")
        cfg = cls(vocab=as_int(raw["vocab"], "vocab", minimum=1), width=as_int(raw["width"], "width", minimum=1),
                  layers=copy.deepcopy(raw["layers"]),
                  max_positions=as_int(raw["max_positions"], "max_positions", minimum=1),
                  norm_eps=as_float(_section(raw, "norm").get("eps", 1e-6), "norm.eps"),
                  logit_softcap=0.0 if cap is None else as_float(cap, "logit_softcap"))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.logit_softcap < 0:
            raise ConfigError(f"logit_softcap must not be negative, got {self.logit_softcap}")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = layer.get("type") if isinstance(layer, dict) else layer
            if kind != "attention":
                raise ConfigError(f"{where}: 'type' must be 'attention', got {kind!r}")
            self._check_mixer(_section(layer, "mixer", where), where + ".mixer")
            self._check_mlp(layer.get("mlp"), where + ".mlp")

    @staticmethod
    def _check_mixer(m: dict, w: str) -> None:
        for key in SIZE_KEYS:
            as_int(m.get(key), f"{w}.{key}", minimum=1)
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{w}: heads must be a multiple of kv_heads")
        if max(2 * m["dim"], m["vdim"]) > 256:
            raise ConfigError(f"{w}: the kernels take dim up to 128 and vdim up to 256, got {m['dim']} and {m['vdim']}")
        as_float(m.get("scale"), f"{w}.scale")
        as_float(m.get("diff"), f"{w}.diff")
        taps = as_int(m.get("conv") or 0, f"{w}.conv", minimum=0)
        if taps > 16:
            raise ConfigError(f"{w}.conv: at most 16 taps, got {taps}")
        mask = m.get("mask")
        if mask is not None:
            if not isinstance(mask, dict):
                raise ConfigError(f"{w}.mask must be a section")
            as_int(mask.get("size"), f"{w}.mask.size", minimum=1)
            as_int(mask.get("keep_first") or 0, f"{w}.mask.keep_first", minimum=0)

    @staticmethod
    def _check_mlp(mlp: Any, w: str) -> None:
        if mlp is None:
            return
        if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
            raise ConfigError(f"{w} must be null or of kind 'dense' or 'moe'")
        if mlp["kind"] == "dense":
            as_int(mlp.get("ff"), f"{w}.ff", minimum=1)
            as_float(mlp.get("limit"), f"{w}.limit")
            return
        router = _section(mlp, "router", w)
        experts = as_int(router.get("experts"), f"{w}.router.experts", minimum=1)
        top = as_int(router.get("top"), f"{w}.router.top", minimum=1)
        if top > experts:
            raise ConfigError(f"{w}.router.top is {top}, there are {experts} experts")
        as_int(_section(mlp, "expert", w).get("ff"), f"{w}.expert.ff", minimum=1)

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "max_positions": self.max_positions, "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(self.layers)}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        return out
