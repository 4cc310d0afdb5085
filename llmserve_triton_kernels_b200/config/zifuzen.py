"""Typed configuration of the Zifuzen design, read from its own config.json keys.

A Zifuzen model embeds tokens and learned positions and runs a list of layers whose norms (layer norms without a bias) stand
behind their parts.  A layer's mixer is the gated delta rule behind short convolutions (``delta`` and ``delta_2``: the same rule,
each with sizes of its own) or grouped-query softmax attention over all earlier positions with per-head norms of q and k and no
rotation (``attention``; with ``kv_from`` it reads the pages that an earlier attention layer wrote).  The feed-forward is dense
(gated by gelu's tanh form, with biases), a mixture of bounded gated experts under a sigmoid router that chooses within groups,
with an optional shared expert, or absent.  The logits pass a soft cap.  Every size and every constant that can differ between
models comes from the dictionary: ``vocab``, ``width``, ``max_positions``, ``embedding.scale``, ``norm.eps``, ``logit_softcap``,
``layers[].type / mixer / mlp``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass

from .llama import ConfigError
from .nurolorn import _need, _positive_int

DELTA_TYPES = ("delta", "delta_2")
MIXER_TYPES = (*DELTA_TYPES, "attention")
MLP_KINDS = ("dense", "moe")


def _heads(m: dict, where: str) -> None:
    for key in ("heads", "kv_heads", "dim", "vdim"):
        _positive_int(_need(m, key, where), f"{where}.{key}")
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"config.json: {where}.heads {m['heads']} is not a multiple of kv_heads {m['kv_heads']}")


def _delta(m: dict, where: str) -> None:
    _heads(m, where)
    if m["dim"] > 256:
        raise ConfigError(f"config.json: {where}.dim {m['dim']}: keys of up to 256 lanes are built")
    if _positive_int(_need(m, "conv", where), f"{where}.conv") > 16:
        raise ConfigError(f"config.json: {where}.conv {m['conv']}: convolutions of up to 16 taps are built")


def _attention(m: dict, where: str, index: int, layers) -> None:
    _heads(m, where)
    _need(m, "scale", where)
    source = m.get("kv_from")
    if source is None:
        return
    if isinstance(source, bool) or not isinstance(source, int) or not 0 <= source < index:
        raise ConfigError(f"config.json: {where}.kv_from {source!r} must name an earlier layer")
    other = layers[source]
    if other.type != "attention" or other.mixer.get("kv_from") is not None:
        raise ConfigError(f"config.json: {where}.kv_from {source}: layer {source} has no keys and values of its own")
    for key in ("kv_heads", "dim", "vdim"):
        if other.mixer.get(key) != m[key]:
            raise ConfigError(f"config.json: {where}.{key} {m[key]} differs from layer {source}'s {other.mixer.get(key)}")


def _mlp(mlp: dict, where: str) -> None:
    kind = _need(mlp, "kind", where)
    if kind not in MLP_KINDS:
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not built; known: {list(MLP_KINDS)}")
    if kind == "dense":
        _positive_int(_need(mlp, "ff", where), f"{where}.ff")
        return
    router = _need(mlp, "router", where)
    r = f"{where}.router"
    experts = _positive_int(_need(router, "experts", r), f"{r}.experts")
    top = _positive_int(_need(router, "top", r), f"{r}.top")
    count, keep = 1, 1
    if router.get("groups"):
        count = _positive_int(_need(router["groups"], "count", f"{r}.groups"), f"{r}.groups.count")
        keep = _positive_int(_need(router["groups"], "keep", f"{r}.groups"), f"{r}.groups.keep")
    if experts % count or keep > count or top > keep * (experts // count):
        raise ConfigError(f"config.json: {r}: {top} of {experts} experts cannot be chosen from {keep} of {count} equal groups")
    for name in ("expert",) + (("shared",) if mlp.get("shared") else ()):
        part = _need(mlp, name, where)
        _positive_int(_need(part, "ff", f"{where}.{name}"), f"{where}.{name}.ff")
        if not float(_need(part, "limit", f"{where}.{name}")) > 0:
            raise ConfigError(f"config.json: {where}.{name}.limit must be positive")


@dataclass(frozen=True)
class ZifuzenLayer:
    type: str  # one of MIXER_TYPES
    mixer: dict  # the mixer's sizes and constants, as config.json gives them
    mlp: dict | None  # {"kind": "dense", "ff"} | {"kind": "moe", "router", "expert", "shared"} | None


@dataclass(frozen=True)
class ZifuzenConfig:
    vocab_size: int  # [vocab]
    width: int  # [width]
    layers: tuple[ZifuzenLayer, ...]  # [layers]
    norm_eps: float  # [norm.eps]
    embedding_scale: float  # [embedding.scale]
    max_positions: int  # [max_positions]: rows of the learned table of positions
    logit_softcap: float | None  # [logit_softcap]; None (the key is absent): the logits as they are

    architecture = "Zifuzen"

    def __post_init__(self) -> None:
        _positive_int(self.vocab_size, "vocab")
        _positive_int(self.width, "width")
        _positive_int(self.max_positions, "max_positions")
        if not self.norm_eps >= 0:
            raise ConfigError("config.json: norm.eps must not be negative")
        if self.logit_softcap is not None and not self.logit_softcap > 0:
            raise ConfigError("config.json: logit_softcap must be positive")
        if not self.layers:
            raise ConfigError("config.json: layers is empty")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if layer.type not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}.type {layer.type!r} is not a mixer of this design; known: {list(MIXER_TYPES)}")
            if layer.type == "attention":
                _attention(layer.mixer, f"{where}.mixer", i, self.layers)
            else:
                _delta(layer.mixer, f"{where}.mixer")
            if layer.mlp is not None:
                _mlp(layer.mlp, f"{where}.mlp")

    @classmethod
    def from_dict(cls, d: dict) -> "ZifuzenConfig":
        layers = []
        for i, entry in enumerate(_need(d, "layers", "the configuration")):
            where = f"layers[{i}]"
            mlp = entry.get("mlp") if isinstance(entry, dict) else None
            layers.append(ZifuzenLayer(_need(entry, "type", where), copy.deepcopy(_need(entry, "mixer", where)), copy.deepcopy(mlp) if mlp else None))
        cap = d.get("logit_softcap")
        return cls(
            vocab_size=_need(d, "vocab", "the configuration"),
            width=_need(d, "width", "the configuration"),
            layers=tuple(layers),
            norm_eps=float(_need(_need(d, "norm", "the configuration"), "eps", "norm")),
            embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
            max_positions=_need(d, "max_positions", "the configuration"),
            logit_softcap=None if cap is None else float(cap),
        )

    def to_dict(self) -> dict:
        """The config.json this configuration is read back from."""
        d = {
            "architecture": self.architecture,
            "embedding": {"scale": self.embedding_scale},
            "layers": [{"type": x.type, "mixer": copy.deepcopy(x.mixer), "mlp": copy.deepcopy(x.mlp)} for x in self.layers],
            "max_positions": self.max_positions,
            "norm": {"eps": self.norm_eps},
            "vocab": self.vocab_size,
            "width": self.width,
        }
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        return d
