"""Configuration of the Givizen decoder, read from its own config.json keys.

    {"architecture": "Givizen", "vocab": V, "width": C, "norm": {"eps": e}, "embedding": {"scale": s},
     "logit_softcap": c, "layers": [{"type": T, "mixer": {...}, "mlp": {...} | null}, ...]}

Mixer types ``attention`` and ``attention_2``, both with ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``,
``mask.size`` (the window; no ``mask``: all earlier keys) and ``q_temp`` (``coef``, ``every``; absent: no temperature);
``attention_2`` also with ``softcap`` (absent: scores are not capped).

``mlp``: ``kind`` "moe" with ``expert`` (``ff``, ``limit``), ``router`` (``experts``, ``top``) and ``shared`` (``ff``,
``limit``; or no ``shared``); or null. Without ``logit_softcap`` the logits are not capped. Every size and constant comes
from the file.
"""

from __future__ import annotations

import copy
import json
from dataclasses import dataclass, field
from pathlib import Path

from .base import ConfigError, ModelConfig, positive, require
from .taredra import _int, _number, _section
from .zefapel import _positive_number

PRESET_DIR = Path(__file__).parent / "presets" / "givizen"

MIXER_TYPES = ("attention", "attention_2")


def _optional_positive(raw: dict, key: str, where: str):
    return None if raw.get(key) is None else _positive_number(raw, key, where)


def _read_mixer(kind: str, raw: dict, where: str) -> dict:
    out = {key: _int(raw, key, where) for key in ("heads", "kv_heads", "dim", "vdim")}
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"config.json: {where}heads ({out['heads']}) must be a multiple of kv_heads ({out['kv_heads']})")
    out["scale"] = _number(raw, "scale", where)
    out["mask"] = out["q_temp"] = None
    if raw.get("mask") is not None:
        out["mask"] = {"size": _int(_section(raw, "mask", where), "size", where + "mask.")}
    if raw.get("q_temp") is not None:
        t, at = _section(raw, "q_temp", where), where + "q_temp."
        every = _positive_number(t, "every", at)
        if every != int(every):
            raise ConfigError(f"config.json: {at}every must be a whole number of positions, got {every!r}")
        out["q_temp"] = {"coef": _number(t, "coef", at), "every": int(every)}
    if kind == "attention_2":
        out["softcap"] = _optional_positive(raw, "softcap", where)
    return out


def _read_expert(raw: dict, where: str) -> dict:
    return {"ff": _int(raw, "ff", where), "limit": _positive_number(raw, "limit", where)}


def _read_mlp(raw, where: str):
    if raw is None:
        return None
    where += "mlp."
    if not isinstance(raw, dict) or raw.get("kind") != "moe":
        raise ConfigError(f"config.json: {where[:-1]} must be null or of kind 'moe', got {raw!r}")
    router, at = _section(raw, "router", where), where + "router."
    r = {"experts": _int(router, "experts", at), "top": _int(router, "top", at)}
    if r["top"] > r["experts"]:
        raise ConfigError(f"config.json: {at}top ({r['top']}) exceeds the {r['experts']} experts a token can choose from")
    out = {"kind": "moe", "expert": _read_expert(_section(raw, "expert", where), where + "expert."), "router": r, "shared": None}
    if raw.get("shared") is not None:
        out["shared"] = _read_expert(_section(raw, "shared", where), where + "shared.")
    return out


def _read_layer(raw: dict, i: int) -> dict:
    where = f"layers[{i}]."
    kind = raw.get("type") if isinstance(raw, dict) else None
    if kind not in MIXER_TYPES:
        raise ConfigError(f"config.json: {where}type '{kind}' is not a mixer of this design {MIXER_TYPES}")
    return {"type": kind, "mixer": _read_mixer(kind, _section(raw, "mixer", where), where + "mixer."),
            "mlp": _read_mlp(raw.get("mlp"), where)}


@dataclass(frozen=True)
class GivizenConfig(ModelConfig):
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_softcap: float | None
    #: one normalised dict per layer (type, mixer, mlp); treated as read-only
    layers: tuple = field(default_factory=tuple)

    architecture = "Givizen"

    @classmethod
    def from_dict(cls, raw: dict) -> "GivizenConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        embedding = raw.get("embedding") if isinstance(raw.get("embedding"), dict) else {}
        cfg = cls(vocab=require(raw, "vocab", int), width=require(raw, "width", int),
                  eps=_number(_section(raw, "norm", ""), "eps", "norm."),
                  embedding_scale=_number(embedding, "scale", "embedding.") if "scale" in embedding else 1.0,
                  logit_softcap=_optional_positive(raw, "logit_softcap", ""),
                  layers=tuple(_read_layer(layer, i) for i, layer in enumerate(layers)))
        positive("vocab", cfg.vocab)
        positive("width", cfg.width)
        if not cfg.eps >= 0:
            raise ConfigError(f"config.json: norm.eps must not be negative, got {cfg.eps!r}")
        return cfg

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embedding_scale}, "logit_softcap": self.logit_softcap,
                "layers": copy.deepcopy(list(self.layers))}

    @classmethod
    def preset_names(cls) -> list[str]:
        return sorted(p.stem for p in PRESET_DIR.glob("*.json"))

    @classmethod
    def preset(cls, name: str) -> "GivizenConfig":
        path = PRESET_DIR / f"{name}.json"
        if not path.is_file():
            raise ConfigError(f"unknown preset '{name}'; known presets: {cls.preset_names()}")
        return cls.from_dict(json.loads(path.read_text()))
