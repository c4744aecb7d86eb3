"""Configuration of the Zefapel decoder, read from its own config.json keys.

    {"architecture": "Zefapel", "vocab": V, "width": C, "norm": {"eps": e}, "embedding": {"scale": s},
     "layers": [{"type": T, "mixer": {...}, "mlp": {...} | null}, ...]}

Mixer types and their keys:

* ``mlstm``: ``heads``, ``dim``, ``vdim``, ``gate_cap``.
* ``gla``: ``heads``, ``dim``, ``vdim``, ``tau``; the rank of the decay's two small matrices is read off the
  checkpoint (``with_tensor_shapes``), or defaults for random weights.
* ``latent_attention``: ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``q_rank``, ``scale``, ``rot`` (``dims``,
  ``base``, ``scaling``: ``factor``, ``original``, ``fast``, ``slow``; absent: frequencies as they are) and, for a layer
  that reads an earlier layer's cached rows, ``kv_from``.

``mlp``: ``kind`` "dense" with ``ff``; or ``kind`` "moe" with ``expert.ff``, ``router`` (``experts``, ``identity``, ``top``,
``groups.count``, ``groups.keep``; without ``identity`` none, without ``groups`` one group) and ``shared.ff`` (or no
``shared``); or null. Every size and constant comes from the file.
"""

from __future__ import annotations

import copy
import json
from dataclasses import dataclass, field, replace
from pathlib import Path

from .base import ConfigError, ModelConfig, positive, require
from .taredra import DEFAULT_DECAY_RANK, _int, _number, _section

PRESET_DIR = Path(__file__).parent / "presets" / "zefapel"

MIXER_TYPES = ("mlstm", "gla", "latent_attention")


def _positive_number(raw: dict, key: str, where: str) -> float:
    value = _number(raw, key, where)
    if not value > 0:
        raise ConfigError(f"config.json: {where}{key} must be positive, got {value!r}")
    return value


def _read_rot(raw: dict, rot_dim: int, where: str) -> dict:
    out = {"dims": _int(raw, "dims", where), "base": _positive_number(raw, "base", where), "scaling": None}
    if out["dims"] != rot_dim or rot_dim % 2:
        raise ConfigError(f"config.json: {where}dims ({out['dims']}) must be even and equal rot_dim ({rot_dim})")
    if raw.get("scaling") is not None:
        s, at = _section(raw, "scaling", where), where + "scaling."
        out["scaling"] = {key: _positive_number(s, key, at) for key in ("factor", "original", "fast", "slow")}
        if out["base"] == 1.0:
            raise ConfigError(f"config.json: {where}base must not be 1 where the frequencies are scaled")
    return out


def _read_mixer(kind: str, raw: dict, where: str) -> dict:
    out = {"heads": _int(raw, "heads", where), "dim": _int(raw, "dim", where), "vdim": _int(raw, "vdim", where)}
    if kind == "mlstm":
        out["gate_cap"] = _positive_number(raw, "gate_cap", where)
    elif kind == "gla":
        out["tau"] = _positive_number(raw, "tau", where)
        if raw.get("rank") is not None:
            out["rank"] = _int(raw, "rank", where)
    else:
        out.update({key: _int(raw, key, where) for key in ("rot_dim", "kv_rank", "q_rank")})
        out["scale"] = _number(raw, "scale", where)
        out["rot"] = _read_rot(_section(raw, "rot", where), out["rot_dim"], where + "rot.")
        src = raw.get("kv_from")
        if src is not None:
            if isinstance(src, bool) or not isinstance(src, int) or src < 0:
                raise ConfigError(f"config.json: {where}kv_from must be a layer's number, got {src!r}")
            out["kv_from"] = src
    return out


def _read_mlp(raw, where: str):
    if raw is None:
        return None
    where += "mlp."
    kind = raw.get("kind") if isinstance(raw, dict) else None
    if kind == "dense":
        return {"kind": "dense", "ff": _int(raw, "ff", where)}
    if kind != "moe":
        raise ConfigError(f"config.json: {where[:-1]} must be null or of kind 'dense' or 'moe', got {raw!r}")
    router, at = _section(raw, "router", where), where + "router."
    identity = router.get("identity") or 0
    if isinstance(identity, bool) or not isinstance(identity, int) or identity < 0:
        raise ConfigError(f"config.json: {at}identity must be a non-negative integer, got {identity!r}")
    r = {"experts": _int(router, "experts", at), "identity": identity, "top": _int(router, "top", at), "groups": None}
    outputs = r["experts"] + identity
    can_take = outputs
    if router.get("groups") is not None:
        g = _section(router, "groups", at)
        count, keep = _int(g, "count", at + "groups."), _int(g, "keep", at + "groups.")
        if outputs % count or keep > count:
            raise ConfigError(f"config.json: {at[:-1]}: {outputs} outputs do not form {count} equal groups of which {keep} are kept")
        r["groups"] = {"count": count, "keep": keep}
        can_take = keep * (outputs // count)
    if r["top"] > can_take:
        raise ConfigError(f"config.json: {at}top ({r['top']}) exceeds the {can_take} outputs a token can choose from")
    out = {"kind": "moe", "expert": {"ff": _int(_section(raw, "expert", where), "ff", where + "expert.")}, "router": r}
    if raw.get("shared") is not None:
        out["shared"] = {"ff": _int(_section(raw, "shared", where), "ff", where + "shared.")}
    return out


def _read_layer(raw: dict, i: int) -> dict:
    where = f"layers[{i}]."
    kind = raw.get("type") if isinstance(raw, dict) else None
    if kind not in MIXER_TYPES:
        raise ConfigError(f"config.json: {where}type '{kind}' is not a mixer of this design {MIXER_TYPES}")
    return {"type": kind, "mixer": _read_mixer(kind, _section(raw, "mixer", where), where + "mixer."),
            "mlp": _read_mlp(raw.get("mlp"), where)}


def _check_shared_rows(layers) -> None:
    """A layer with ``kv_from`` reads the rows of an earlier latent layer that keeps its own, made alike."""
    for i, layer in enumerate(layers):
        src = layer["mixer"].get("kv_from")
        if src is None:
            continue
        m, where = layer["mixer"], f"config.json: layers[{i}].mixer.kv_from"
        if src >= i or layers[src]["type"] != "latent_attention" or "kv_from" in layers[src]["mixer"]:
            raise ConfigError(f"{where} must name an earlier latent_attention layer that keeps rows of its own, got {src}")
        s = layers[src]["mixer"]
        if any(m[key] != s[key] for key in ("kv_rank", "rot_dim", "rot")):
            raise ConfigError(f"{where}: kv_rank, rot_dim and rot must equal those of layer {src}")


@dataclass(frozen=True)
class ZefapelConfig(ModelConfig):
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    #: one normalised dict per layer (type, mixer, mlp); treated as read-only
    layers: tuple = field(default_factory=tuple)

    architecture = "Zefapel"

    @classmethod
    def from_dict(cls, raw: dict) -> "ZefapelConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        embedding = raw.get("embedding") if isinstance(raw.get("embedding"), dict) else {}
        cfg = cls(vocab=require(raw, "vocab", int), width=require(raw, "width", int),
                  eps=_number(_section(raw, "norm", ""), "eps", "norm."),
                  embedding_scale=_number(embedding, "scale", "embedding.") if "scale" in embedding else 1.0,
                  layers=tuple(_read_layer(layer, i) for i, layer in enumerate(layers)))
        positive("vocab", cfg.vocab)
        positive("width", cfg.width)
        if not cfg.eps >= 0:
            raise ConfigError(f"config.json: norm.eps must not be negative, got {cfg.eps!r}")
        _check_shared_rows(cfg.layers)
        return cfg

    def with_tensor_shapes(self, shapes: dict) -> "ZefapelConfig":
        """The decays' rank is the first size of each ``gla`` layer's ``mix.a1``."""
        layers = copy.deepcopy(list(self.layers))
        for i, layer in enumerate(layers):
            shape = shapes.get(f"l{i}.mix.a1")
            if layer["type"] == "gla" and shape is not None:
                layer["mixer"]["rank"] = int(shape[0])
        return replace(self, layers=tuple(layers))

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embedding_scale}, "layers": copy.deepcopy(list(self.layers))}

    @classmethod
    def preset_names(cls) -> list[str]:
        return sorted(p.stem for p in PRESET_DIR.glob("*.json"))

    @classmethod
    def preset(cls, name: str) -> "ZefapelConfig":
        path = PRESET_DIR / f"{name}.json"
        if not path.is_file():
            raise ConfigError(f"unknown preset '{name}'; known presets: {cls.preset_names()}")
        return cls.from_dict(json.loads(path.read_text()))


def decay_rank(mixer: dict) -> int:
    return int(mixer.get("rank", DEFAULT_DECAY_RANK))
