"""A model as data: layers named by their parts, and the order in which they run."""

from __future__ import annotations

from dataclasses import dataclass
from types import MappingProxyType
from typing import Mapping

from ..parts.base import PartSpec


class LayerSpec:
    """One layer: the kind of block that arranges it, and the parts that block asks for, by role.

    Which roles there are is the block kind's business (``Block.roles``: role -> part category): the pre-norm block
    has ``mixer_norm, mixer, ff_norm, feed_forward``; a block with norms after its parts as well, or with one norm and
    two parallel parts, names other roles and is built from the same ``LayerSpec(block, role=spec, ...)``."""

    __slots__ = ("block", "parts")

    def __init__(self, block: PartSpec, parts: Mapping[str, PartSpec] | None = None, **roles: PartSpec):
        object.__setattr__(self, "block", block)
        object.__setattr__(self, "parts", MappingProxyType({**(parts or {}), **roles}))

    def __setattr__(self, name, value):
        raise AttributeError("a LayerSpec is not changed after it is made")

    def __getattr__(self, role: str) -> PartSpec:  # spec.mixer, spec.ff_norm, ...
        try:
            return self.parts[role]
        except KeyError:
            raise AttributeError(role) from None

    def replace(self, block: PartSpec | None = None, **roles: PartSpec) -> "LayerSpec":
        """A copy with another block or other parts in the named roles."""
        return LayerSpec(block or self.block, {**self.parts, **roles})

    def __eq__(self, other) -> bool:
        return isinstance(other, LayerSpec) and self.block == other.block and dict(self.parts) == dict(other.parts)

    def __hash__(self) -> int:
        return hash((self.block.kind, tuple(self.parts)))

    def __repr__(self) -> str:
        return f"LayerSpec({self.block!r}, {dict(self.parts)!r})"


@dataclass(frozen=True)
class LayerRun:
    """One entry of the execution order.

    ``layer`` indexes ``ModelPlan.layers`` and may appear in several entries (the same weights
    run twice; each entry then keeps a cache of its own).  ``cache_of`` names an earlier entry
    of the order whose cache this entry reads instead of keeping one (shared keys and values).
    """

    layer: int
    cache_of: int | None = None


@dataclass(frozen=True)
class Injection:
    """What the residual stream takes up before an entry of the order runs (after what the entry in front left has
    been added): the token embeddings once more, and/or row ``row`` of the tensor ``vector`` ``[rows, hidden]``.
    A stretch of layers that runs several times with the same weights marks its passes this way."""

    before: int  # index into ``ModelPlan.schedule``
    add_embedding: bool = False
    vector: str | None = None  # name of a tensor declared in ``ModelPlan.extra_tensors``
    row: int = 0


@dataclass(frozen=True)
class ModelPlan:
    hidden_size: int
    vocab_size: int
    max_positions: int | None  # None: no limit of the model's own (the cache's room bounds a request)
    embedding: str  # tensor name of the token table [vocab, hidden]
    layers: tuple[LayerSpec, ...]
    schedule: tuple[LayerRun, ...]
    final_norm: PartSpec
    head: str | None  # tensor name of the output matrix [vocab, hidden]; None: the token table
    ignored: tuple[str, ...] = ()  # names a checkpoint may carry that the model does not read (e.g. a copy of a tied head)
    injections: tuple[Injection, ...] = ()
    extra_tensors: tuple[tuple[str, tuple[int, ...]], ...] = ()  # (name, shape) of tensors that belong to no part
    logit_scale: float = 1.0  # the logits are the output matrix's product times this
    embedding_scale: float = 1.0  # the residual stream starts as the tokens' rows of the table times this
    positions: str | None = None  # tensor name of a table [max_positions, hidden] whose row p is added to the embedding of a token at position p
    logit_softcap: float | None = None  # the logits z (after logit_scale) become cap * tanh(z / cap)
    streams: int | None = None  # the residual stream is kept in this many copies [streams, N, hidden], all equal at the start (None: one plain stream)

    def __post_init__(self) -> None:
        for i, run in enumerate(self.schedule):
            if not 0 <= run.layer < len(self.layers):
                raise ValueError(f"schedule entry {i} names layer {run.layer}, of {len(self.layers)}")
            if run.cache_of is not None:
                if not 0 <= run.cache_of < i:
                    raise ValueError(f"schedule entry {i} reads the cache of entry {run.cache_of}, which is not earlier")
                if self.schedule[run.cache_of].cache_of is not None:
                    raise ValueError(f"schedule entry {i} reads the cache of entry {run.cache_of}, which keeps none itself")
        if self.streams is not None and (self.streams < 1 or self.injections):
            raise ValueError("a stream kept in copies needs at least one copy, and takes nothing up between its layers")
        if self.positions is not None and (self.max_positions is None or self.streams is not None):
            raise ValueError("a table of positions has a row for each of max_positions places, and feeds one plain stream")
        declared = {name for name, _ in self.extra_tensors}
        seen = set()
        for inj in self.injections:
            if not 0 <= inj.before < len(self.schedule) or inj.before in seen:
                raise ValueError(f"an injection names entry {inj.before} of {len(self.schedule)}, or an entry twice")
            seen.add(inj.before)
            if inj.vector is not None and inj.vector not in declared:
                raise ValueError(f"an injection reads the tensor {inj.vector!r}, which the plan does not declare")
