"""Typed configuration of the Pefedra design, read from its own config.json keys.

A Pefedra model is a list of layers in which mixer and feed-forward read the same stream side by side, each behind a norm of its
own, with a token shift on what the mixer reads.  A layer's mixer is one of two kinds of grouped-query softmax attention over a
sliding window: ``attention`` (two score maps a head over the same values, the second subtracted from the first) and
``attention_2`` (q and k normed over their whole projections, values that are rotated with their positions and turned back behind
the sum, a sigmoid gate per head).  The feed-forward is dense or absent.  Every size and every constant that can differ between
models comes from the dictionary: ``vocab``, ``width``, ``embedding.scale``, ``norm.eps``, ``layers[].type / mixer / mlp``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass

from .llama import ConfigError
from .nurolorn import _need, _positive_int

MIXER_TYPES = ("attention", "attention_2")
MLP_KINDS = ("dense",)


def _rot(rot, most: int, where: str) -> None:
    dims = _need(rot, "dims", where)
    if isinstance(dims, bool) or not isinstance(dims, int) or dims % 2 or not 0 <= dims <= most:
        raise ConfigError(f"config.json: {where}.dims {dims!r} must be even and at most {most}")
    _need(rot, "base", where)
    scaling = rot.get("scaling")
    if scaling and not float(_need(scaling, "factor", f"{where}.scaling")) > 0:
        raise ConfigError(f"config.json: {where}.scaling.factor must be positive")


def _mixer(kind: str, m: dict, where: str) -> None:
    for key in ("heads", "kv_heads", "dim", "vdim"):
        _positive_int(_need(m, key, where), f"{where}.{key}")
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"config.json: {where}.heads {m['heads']} is not a multiple of kv_heads {m['kv_heads']}")
    _need(m, "scale", where)
    _positive_int(_need(_need(m, "mask", where), "size", f"{where}.mask"), f"{where}.mask.size")
    _rot(_need(m, "rot", where), m["dim"], f"{where}.rot")
    if kind == "attention":
        _need(m, "diff", where)
    elif m["vdim"] % 2:
        raise ConfigError(f"config.json: {where}.vdim {m['vdim']}: rotated values have an even number of lanes")


@dataclass(frozen=True)
class PefedraLayer:
    type: str  # one of MIXER_TYPES
    mixer: dict  # the mixer's sizes and constants, as config.json gives them
    mlp: dict | None  # {"kind": "dense", "ff"} | None


@dataclass(frozen=True)
class PefedraConfig:
    vocab_size: int  # [vocab]
    width: int  # [width]
    layers: tuple[PefedraLayer, ...]  # [layers]
    norm_eps: float  # [norm.eps]
    embedding_scale: float  # [embedding.scale]
    max_positions: int | None = None  # not a key of the design: an engine may bound a request's length with it

    architecture = "Pefedra"

    def __post_init__(self) -> None:
        _positive_int(self.vocab_size, "vocab")
        _positive_int(self.width, "width")
        if not self.norm_eps >= 0:
            raise ConfigError("config.json: norm.eps must not be negative")
        if not self.layers:
            raise ConfigError("config.json: layers is empty")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if layer.type not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}.type {layer.type!r} is not a mixer of this design; known: {list(MIXER_TYPES)}")
            _mixer(layer.type, layer.mixer, f"{where}.mixer")
            if layer.mlp is not None:
                kind = _need(layer.mlp, "kind", f"{where}.mlp")
                if kind not in MLP_KINDS:
                    raise ConfigError(f"config.json: {where}.mlp.kind {kind!r} is not built; known: {list(MLP_KINDS)}")
                _positive_int(_need(layer.mlp, "ff", f"{where}.mlp"), f"{where}.mlp.ff")

    @classmethod
    def from_dict(cls, d: dict) -> "PefedraConfig":
        layers = []
        for i, entry in enumerate(_need(d, "layers", "the configuration")):
            where = f"layers[{i}]"
            mlp = entry.get("mlp") if isinstance(entry, dict) else None
            layers.append(PefedraLayer(_need(entry, "type", where), copy.deepcopy(_need(entry, "mixer", where)), copy.deepcopy(mlp) if mlp else None))
        limit = d.get("max_positions")
        return cls(
            vocab_size=_need(d, "vocab", "the configuration"),
            width=_need(d, "width", "the configuration"),
            layers=tuple(layers),
            norm_eps=float(_need(_need(d, "norm", "the configuration"), "eps", "norm")),
            embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
            max_positions=None if limit is None else int(limit),
        )

    def to_dict(self) -> dict:
        """The config.json this configuration is read back from."""
        d = {
            "architecture": self.architecture,
            "embedding": {"scale": self.embedding_scale},
            "layers": [{"type": x.type, "mixer": copy.deepcopy(x.mixer), "mlp": copy.deepcopy(x.mlp)} for x in self.layers],
            "norm": {"eps": self.norm_eps},
            "vocab": self.vocab_size,
            "width": self.width,
        }
        if self.max_positions is not None:
            d["max_positions"] = self.max_positions
        return d
