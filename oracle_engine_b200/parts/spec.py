"""The data description of a model: which parts make each layer, and in what order the
layers run.

An architecture's `build_spec(config)` returns a `ModelSpec`.  Nothing below it knows
which model it is in: every part gets its sizes and constants from its `PartSpec`.

* `PartSpec(kind, params)` names a registered part (parts/registry.py) and its parameters.
* `LayerSpec` puts a mixer, a feed-forward and their norms together in an arrangement
  (`block`), under a tensor-name prefix.  Layers may differ from one another.
* `ModelSpec.schedule` is the order in which layers run: a list of `ScheduleEntry`.  An
  entry may name a layer that another entry also names (the weights are shared; each entry
  still has a cache of its own), and `cache_from` lets an entry read the cache that an
  earlier entry wrote instead of writing one (it then computes no keys or values), and `before` names a part
  of `ModelSpec.stream_parts` that works on the stream right before the entry's layer.

The reference has one fixed arrangement, x += Attn(RMSNorm(x)); x += FFN(RMSNorm(x)),
L times (core/model.cpp:361-474); here that order is the data a Llama spec holds.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Optional


@dataclass(frozen=True)
class TensorDecl:
    """A weight a part needs: full name in the file, shape, and how random weights fill it
    ("normal": N(0, std); "ones_normal": 1 + N(0, norm_std)).  A size of -1 is one that only the file gives."""
    name: str
    shape: tuple[int, ...]
    init: str = "normal"


@dataclass(frozen=True)
class PartSpec:
    kind: str
    params: dict = field(default_factory=dict)


@dataclass(frozen=True)
class LayerSpec:
    prefix: str                        # e.g. "model.layers.3."
    mixer: PartSpec
    feed_forward: Optional[PartSpec]
    mixer_norm: PartSpec
    ffn_norm: Optional[PartSpec]
    block: str = "pre_norm"            # arrangement of the four (parts/block.py)
    block_params: dict = field(default_factory=dict)   # an arrangement's own constants and tensor names, if it has any


@dataclass(frozen=True)
class ScheduleEntry:
    layer: int                         # index into ModelSpec.layers
    cache_from: Optional[int] = None   # index of an earlier schedule entry whose cache is read
    # (name in ModelSpec.stream_parts, ((argument, value), ...)): a part that works on the stream right before this
    # entry's layer, e.g. what a looped group of layers adds when a pass begins
    before: Optional[tuple] = None


@dataclass(frozen=True)
class CacheNeed:
    """What a mixer keeps per token in the paged cache.

    `tensors`: ((name, per-token shape), ...), one entry per tensor the mixer keeps.  A tensor
    whose per-token shape is (a, ..., z) is stored per page as [a, ..., PAGE, z] (the page's
    tokens run along the last but one axis, so that a token's innermost vector is contiguous
    and a page of one outer index is one block).  Attention keeps one tensor "kv" of shape
    (2, kv_heads, head_dim); a mixer that keeps one latent vector per token would declare
    (("latent", (rank,)),), keys and values of different widths two tensors.
    `kind`: "full" (every position), "window" (the last `window` of them; older pages are
    given back) or "chunk" (those of the query's own chunk of `window` positions, counted from
    position 0; the pages of finished chunks are given back).  `also`: (kind, window) pairs of
    further readers of the same rows: what any of them still sees is kept.
    Entries with equal needs share one group of storage and page tables."""
    kind: str
    tensors: tuple
    window: int = 0
    also: tuple = ()

    def first_position(self, pos: int) -> int:
        """The oldest position that a query at `pos`, or at any later one, still reads."""
        first = pos
        for kind, n in ((self.kind, self.window),) + self.also:
            if kind == "full":
                return 0
            first = min(first, max(0, pos - n + 1) if kind == "window" else pos - pos % n)
        return first

    def joined(self, other: "CacheNeed") -> "CacheNeed":
        """The need of rows that both this need's owner and the mixer of `other` read."""
        mine, theirs = ((self.kind, self.window),) + self.also, ((other.kind, other.window),) + other.also
        if set(theirs) <= set(mine):
            return self
        if any(kind == "full" for kind, _ in mine + theirs):
            return CacheNeed("full", self.tensors)
        rest = sorted(set(mine + theirs) - {(self.kind, self.window)})
        return CacheNeed(self.kind, self.tensors, self.window, tuple(rest))

    def elements_per_token(self) -> int:
        n = 0
        for _, shape in self.tensors:
            e = 1
            for d in shape:
                e *= int(d)
            n += e
        return n


def span_need(tensors: tuple, span: int) -> CacheNeed:
    """The need of an attention whose mask is `span` as the kernels take it (csrc/common.cuh: oe_first_key): 0 every
    key, n > 0 the last n keys, -n the keys of the query's own chunk of n."""
    return CacheNeed("window" if span > 0 else "chunk" if span < 0 else "full", tensors, abs(int(span)))


def attention_cache_need(kv_heads: int, head_dim: int, span: int = 0) -> CacheNeed:
    """Keys and values of grouped-query attention: one tensor "kv", per page [2, kv_heads, PAGE, head_dim]."""
    return span_need((("kv", (2, int(kv_heads), int(head_dim))),), span)


def mask_span(window, chunk) -> int:
    """An attention's `window` and `chunk` parameters (0 or None: no such mask) as one span."""
    window, chunk = int(window or 0), int(chunk or 0)
    if window < 0 or chunk < 0 or (window and chunk):
        raise ValueError(f"an attention has a window or chunks of a positive size, not both: {window}, {chunk}")
    return window if window else -chunk


def visible_keys(span: int, context: int) -> int:
    """How many keys the newest of `context` tokens sees."""
    return min(context, span) if span > 0 else (context - 1) % -span + 1 if span < 0 else context


def visible_pairs(span: int, start: int, count: int) -> float:
    """The (query, key) pairs of `count` tokens at positions start .. start + count - 1."""
    tri = lambda n: n * (n + 1) / 2.0                                    # noqa: E731
    upto = lambda n: tri(n) if not span else \
        tri(min(n, span)) + span * max(0, n - span) if span > 0 else \
        (n // -span) * tri(-span) + tri(n % -span)                       # noqa: E731
    return upto(start + count) - upto(start)


@dataclass(frozen=True)
class StateNeed:
    """Per-sequence state of fixed size that a part keeps: one tensor of `shape` per
    sequence, zeroed when a sequence starts."""
    shape: tuple[int, ...]
    dtype: Any                         # torch dtype


@dataclass(frozen=True)
class ModelSpec:
    architecture: str
    hidden_size: int
    vocab_size: int
    max_positions: int
    embedding: PartSpec
    final_norm: PartSpec
    head: PartSpec
    positions: dict                    # name -> PartSpec of a position encoding
    layers: tuple
    schedule: tuple
    stop_ids: tuple = ()
    bos_id: Optional[int] = None
    ignored_tensors: tuple = ()        # name suffixes a file may hold that the model does not read
    stream_parts: dict = field(default_factory=dict)   # name -> PartSpec of a part that schedule entries run `before` their layer

    def __post_init__(self):
        for i, e in enumerate(self.schedule):
            if not 0 <= e.layer < len(self.layers):
                raise ValueError(f"schedule[{i}] names layer {e.layer}, there are {len(self.layers)}")
            if e.before is not None and e.before[0] not in self.stream_parts:
                raise ValueError(f"schedule[{i}].before names the stream part {e.before[0]!r}, which the model does not have")
            if e.cache_from is not None:
                if not 0 <= e.cache_from < i:
                    raise ValueError(f"schedule[{i}].cache_from must name an earlier entry, got {e.cache_from}")
                if self.schedule[e.cache_from].cache_from is not None:
                    raise ValueError(f"schedule[{i}].cache_from names an entry that owns no cache")
