"""Architecture-independent description of a decoder.

A model family turns its own ``config.json`` into a :class:`ModelSpec`: plain
data that says, layer by layer, which mixer, feed-forward, norms and position
encoding to build, with every size and constant as a parameter, and in which
order the layers run. Nothing below this file knows a family's name; the
parts are built from the spec by kind (``metallix_b200.parts.registry``).

The reference engine hard-codes one arrangement in
``crates/models/qwen/src/forward.rs:1856-1922`` (pre-norm attention, residual,
pre-norm SwiGLU, residual). Here the same arrangement is one value of
``LayerSpec.block``, and the loop over layers (``forward.rs:1562-1582``) is the
``order`` list.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Tuple


@dataclass(frozen=True)
class PartSpec:
    """One buildable part: a registered ``kind`` and its parameters.

    ``params`` holds sizes, constants and tensor names; a part reads nothing
    else. Two parts of the same kind with different params may sit in
    different layers of one model.
    """

    kind: str
    params: Mapping[str, Any] = field(default_factory=dict)

    def get(self, key: str, default: Any = None) -> Any:
        return self.params.get(key, default)

    def __getitem__(self, key: str) -> Any:
        return self.params[key]


@dataclass(frozen=True)
class LayerSpec:
    """One decoder layer: what it is made of and how the pieces are arranged."""

    name: str  # tensor-name prefix, e.g. "model.layers.3"
    block: PartSpec  # the arrangement (pre-norm residual, ...)
    mixer: PartSpec
    feed_forward: Optional[PartSpec]        # None: the layer has no feed-forward
    mixer_norm: PartSpec
    feed_forward_norm: Optional[PartSpec]
    # Norms a sublayer's output passes before it joins the residual stream
    # (an arrangement that has none ignores them).
    mixer_post_norm: Optional[PartSpec] = None
    feed_forward_post_norm: Optional[PartSpec] = None


@dataclass(frozen=True)
class LayerRun:
    """One entry of the execution order.

    ``layer`` indexes ``ModelSpec.layers`` (a layer may be named twice; its
    second run then needs a cache entry of its own, any unused index).
    ``cache`` is the cache entry the mixer uses; by default a layer owns the
    entry with its own index. ``write_cache=False`` lets a layer read the
    entry another layer has written in the same step without writing to it.
    """

    layer: int
    cache: Optional[int] = None
    write_cache: bool = True
    join: Optional[int] = None      # which of ModelSpec.joins acts on the residual stream right before this run
    turn: int = 0                   # ... and for which time, for a join with parameters per turn

    def cache_entry(self) -> int:
        return self.layer if self.cache is None else self.cache


@dataclass(frozen=True)
class CacheNeed:
    """What one cache entry needs from the cache manager.

    ``kind == "kv_pages"``: keys and values of ``kv_heads`` heads of width
    ``head_dim`` for every position (``window is None``) or for the last
    ``window`` positions; with ``chunk`` only the positions of the chunk of
    that many positions (counted from position 0) the next query lies in are
    ever read again; the first ``keep`` positions of a sequence are kept beside
    either. ``planes`` is 2 for keys and values, 1 for a pool with
    one row per position that serves as both (a latent that all heads share).
    ``kind == "state"``: ``state_shape`` values of fixed
    size per request, zeroed when the request is admitted. ``kind == "none"``:
    the mixer keeps nothing between steps. ``kind == "several"``: a mixer made
    of mixers; ``members`` are their needs, in the mixer's own order.
    """

    kind: str
    kv_heads: int = 0
    head_dim: int = 0
    window: Optional[int] = None
    chunk: Optional[int] = None
    state_shape: Tuple[int, ...] = ()
    state_dtype: str = "float32"
    planes: int = 2
    members: Tuple["CacheNeed", ...] = ()
    keep: int = 0

    def group_key(self) -> tuple:
        return (self.kind, self.kv_heads, self.head_dim, self.window, self.chunk, self.keep,
                tuple(self.state_shape), self.state_dtype, self.planes,
                tuple(member.group_key() for member in self.members))

    def flat(self) -> Tuple["CacheNeed", ...]:
        """The needs that take memory: this one, or a mixer-of-mixers' members (to any depth)."""
        if self.kind != "several":
            return (self,)
        return tuple(need for member in self.members for need in member.flat())

    def has_state(self) -> bool:
        """Whether a step advances something that running it twice would advance twice."""
        return any(need.kind == "state" for need in self.flat())


@dataclass(frozen=True)
class ModelSpec:
    """Everything the engine needs to build a decoder, and nothing family-specific."""

    architecture: str
    hidden_size: int
    vocab_size: int
    max_positions: int
    embedding: PartSpec
    layers: Tuple[LayerSpec, ...]
    order: Tuple[LayerRun, ...]
    final_norm: PartSpec
    head: PartSpec
    # 0: one residual stream [tokens, hidden]. s >= 1: s copies of it,
    # [tokens, s, hidden], all equal to the embedding at the start and summed at
    # the end, which blocks of a hyper-connection arrangement read and write.
    streams: int = 0
    # What may happen to the residual stream ahead of a layer run (``LayerRun.join``).
    joins: Tuple[PartSpec, ...] = ()

    def num_cache_entries(self) -> int:
        return max(run.cache_entry() for run in self.order) + 1

    def validate(self) -> None:
        if not self.layers:
            raise ValueError("a model needs at least one layer")
        written = set()
        for run in self.order:
            if not 0 <= run.layer < len(self.layers):
                raise ValueError(f"order names layer {run.layer}, the model has {len(self.layers)}")
            if run.join is not None and not (0 <= run.join < len(self.joins) and self.streams == 0):
                raise ValueError(f"order names join {run.join}, the model has {len(self.joins)} and {self.streams} streams")
            entry = run.cache_entry()
            if entry < 0:
                raise ValueError(f"order names cache entry {entry}")
            if run.write_cache:
                written.add(entry)
            elif entry not in written:
                raise ValueError(
                    f"layer {run.layer} reads cache entry {entry} before any layer has written it")
