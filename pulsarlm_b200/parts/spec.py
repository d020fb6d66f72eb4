"""A model as data: which parts, with which sizes, reading which tensors, in which order.

An architecture's `describe(config)` returns a ModelSpec. The generic model
(pulsarlm_b200/models/model.py) builds parts from it through the part
registries; no part learns which architecture it sits in.
"""

from __future__ import annotations

import dataclasses
from typing import Any


@dataclasses.dataclass
class PartSpec:
    """One part: `kind` selects the class in its registry, `params` are its sizes
    and constants, `tensors` maps the part's own role names (e.g. "q", "gate")
    to tensor names in the checkpoint. A role mapped to None is absent (e.g. a
    tied head has no tensor of its own)."""

    kind: str
    params: dict[str, Any] = dataclasses.field(default_factory=dict)
    tensors: dict[str, str | None] = dataclasses.field(default_factory=dict)


@dataclasses.dataclass
class LayerSpec:
    """One layer: an arrangement (`block`, e.g. "pre_norm") of a mixer, a
    feed-forward (None where the arrangement allows a layer without one) and the norms
    the arrangement names. `extras`: whatever else the arrangement takes (constants,
    PartSpecs of further parts), by the names it documents."""

    block: str
    mixer: PartSpec
    feed_forward: PartSpec | None
    norms: dict[str, PartSpec]
    extras: dict[str, Any] = dataclasses.field(default_factory=dict)


@dataclasses.dataclass
class ModelSpec:
    """The whole model. `order` lists layer indices in the order they run; an
    index may appear twice (the layer then runs twice with the same weights and
    cache). A mixer whose params hold `cache_from = k` reads (and does not
    write) the cache of layer k. `cache_per_run`: every entry of `order` keeps a
    cache or state of its own (a layer that runs twice then has two, one per run),
    and the cache manager is asked run by run instead of layer by layer.
    `rejoin_runs`: places in `order` before which the embedding's output (the
    stream as it entered the first layer) is added to the stream again. `join` with
    `join_runs`: a part of the "join" registry that makes a new stream of the stream and
    the embedding's output before those places in `order` (the first place too, if listed).
    `max_positions`: the most tokens a sequence can hold, for a model with a table of positions
    (None: no such bound)."""

    hidden_size: int
    vocab_size: int
    embedding: PartSpec
    layers: list[LayerSpec]
    order: list[int]
    final_norm: PartSpec
    head: PartSpec
    eos_token_ids: tuple[int, ...] = ()
    max_position_embeddings: int | None = None
    max_positions: int | None = None
    cache_per_run: bool = False
    rejoin_runs: tuple[int, ...] = ()
    join: PartSpec | None = None
    join_runs: tuple[int, ...] = ()


@dataclasses.dataclass(frozen=True)
class TensorNeed:
    """What a part expects of one checkpoint tensor. `role` is "matrix" for
    operands of matrix products and embedding tables (converted to the engine's
    dtype) or "vector" for scales and the like (a tensor stored in 32-bit stays
    32-bit), "offset" for biases and other vectors around zero (kept like "vector";
    random weights draw them around 0 instead of 1), or "ignored" for a tensor that may
    be stored but is not read. `optional` tensors may be missing."""

    shape: tuple[int, ...]
    role: str = "matrix"
    optional: bool = False


@dataclasses.dataclass(frozen=True)
class KVCacheNeed:
    """A mixer that keeps keys and values: per token `n_kv_heads * head_dim` keys
    and as many values. `window` = None keeps every token; a number keeps only the
    last `window` tokens readable, and pages wholly before them are given back;
    `keep_first` tokens at a sequence's start stay readable besides (their pages stay).
    `n_heads` is the number of query heads that read the cache; the cache manager
    sizes the optional per-page attention-mass accumulators by it. `planes` = 2 keeps
    keys and values; 1 keeps one row per token that serves as both (a mixer that caches
    a shared latent)."""

    n_kv_heads: int
    head_dim: int
    window: int | None = None
    n_heads: int = 0
    planes: int = 2
    keep_first: int = 0


@dataclasses.dataclass(frozen=True)
class StateNeed:
    """A part that keeps a state of fixed size per request: `shape` elements of
    `dtype` ("float32", "bfloat16", "int32", or "engine" for the engine's dtype), zeroed
    when a request gets its slot."""

    shape: tuple[int, ...]
    dtype: str = "float32"
