"""The generic model: parts built from a ModelSpec and run in the spec's order.

Nothing here is specific to an architecture. The model owns no cache; the cache
manager asks `cache_needs()` what each layer wants and hands bindings back
through `bind_caches()`.
"""

from __future__ import annotations

import dataclasses

import torch

from ..parts import attention, basic, block  # noqa: F401  (registers the built-in parts)
from ..parts.registry import BuildContext, build_part, part_class
from ..parts.spec import ModelSpec, TensorNeed


@dataclasses.dataclass
class StepBatch:
    """One step's tokens, on the device.

    tokens, pos, entry: int32 [T]; token t is `tokens[t]` at position `pos[t]` of
    the request in batch entry `entry[t]`. tables[g]: int32 [entries, width], the
    block-table rows of cache group g for this step's entries. slots: int32
    [entries], each entry's state slot. want_rows: int32 [R], indices into the T
    tokens whose logits are wanted (None: none). status: int32 [1] that kernels
    OR error bits into. Entries of a single token come first: the leading `n_decode`
    tokens are each the one token of their entry. The host_* fields repeat sizes
    for kernels' launchers.
    """

    tokens: torch.Tensor
    pos: torch.Tensor
    entry: torch.Tensor
    tables: dict[int, torch.Tensor]
    slots: torch.Tensor
    want_rows: torch.Tensor | None
    status: torch.Tensor
    n_tokens: int
    n_entries: int
    n_decode: int = 0
    host_query_lens: list[int] = dataclasses.field(default_factory=list)
    host_context_lens: list[int] = dataclasses.field(default_factory=list)
    extras: dict = dataclasses.field(default_factory=dict)
    # What the parts planned for this step on the host (see HostStep): plans[key][name]
    # is a device tensor for every array a part's plan_step returned under `name`, and
    # the value itself for everything else. `key` is the part's plan_key().
    plans: dict = dataclasses.field(default_factory=dict)


@dataclasses.dataclass
class HostStep:
    """What the host knows of a step before it runs: the sizes of its entries, in batch
    order (entries of one token first). Parts that need index arrays of their own for
    a step (tile lists, chunk boundaries, expert offsets) build them from this in
    `plan_step`; the step function stages what they return with its own arrays and
    hands it back in `StepBatch.plans`.

    query_lens[e]: tokens of entry e in this step. context_lens[e]: tokens its
    request holds after the step. first_rows[e]: row of its first token among the
    step's tokens. A step that is captured once and replayed (`fixed_shape`) is
    planned anew before every replay: the arrays a part returns must then have shapes
    that depend only on n_entries and context_bound (the most tokens any entry of a
    replay may hold), and what it returns besides arrays is kept from the first call,
    so it must depend on nothing else either. A part that wants different kernels for
    different replays of one shape (say, for requests of equal and of unequal lengths)
    answers `plan_variant(step)` with a hashable value: replays whose values differ get
    captures of their own, and `variants[part.plan_key()]` holds the value the capture
    at hand was made for."""

    n_entries: int
    n_tokens: int
    n_decode: int
    query_lens: list[int]
    context_lens: list[int]
    first_rows: list[int]
    page_size: int
    fixed_shape: bool = False
    context_bound: int | None = None
    variants: dict = dataclasses.field(default_factory=dict)


def _all_part_specs(spec: ModelSpec):
    yield "embedding", spec.embedding
    for layer in spec.layers:
        yield from part_class("block", layer.block).part_specs(layer)
    if spec.join is not None:
        yield "join", spec.join
    yield "norm", spec.final_norm
    yield "head", spec.head


def tensor_needs_of(spec: ModelSpec) -> dict[str, TensorNeed]:
    """Every checkpoint tensor the model's parts need, by name. A name two parts
    ask for must be asked for with the same shape."""
    needs: dict[str, TensorNeed] = {}
    for kind, part_spec in _all_part_specs(spec):
        for name, need in part_class(kind, part_spec.kind).tensor_needs(part_spec).items():
            if name in needs and needs[name].shape != need.shape:
                raise ValueError(f"tensor {name!r} is needed with shapes {needs[name].shape} and {need.shape}")
            needs.setdefault(name, need)
    return needs


class Model:
    """Embedding, blocks in `spec.order`, final norm, head."""

    def __init__(self, spec: ModelSpec, dtype: torch.dtype, device: torch.device):
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"engine dtype must be float32 or bfloat16, got {dtype}")
        self.spec = spec
        self.ctx = BuildContext(dtype=dtype, device=torch.device(device))
        for index in spec.order:
            if not 0 <= index < len(spec.layers):
                raise ValueError(f"layer order names layer {index}, but there are {len(spec.layers)} layers")
        self.embedding = build_part("embedding", spec.embedding, self.ctx)
        self.blocks = [part_class("block", layer.block)(layer, self.ctx) for layer in spec.layers]
        self.final_norm = build_part("norm", spec.final_norm, self.ctx)
        self.head = build_part("head", spec.head, self.ctx)
        self.join = build_part("join", spec.join, self.ctx) if spec.join is not None else None
        self.loaded = False
        # The cache units, in the order the cache manager hears of them: one per layer, or
        # (spec.cache_per_run) one per entry of the order. `_unit_layer[u]` is the layer of unit u.
        self._unit_layer = list(spec.order) if spec.cache_per_run else list(range(len(spec.layers)))
        # Parts outside the layers that keep something per request (an embedding that remembers a
        # request's last token): their needs follow the layers' in `cache_needs()`.
        self._own_holders = [part for part in (self.embedding,) if hasattr(part, "cache_need")]
        self._run_bindings: list | None = None
        self._rejoin = frozenset(int(r) for r in spec.rejoin_runs)
        for r in self._rejoin:
            if not 0 < r < len(spec.order):
                raise ValueError(f"the embedding cannot rejoin the stream before run {r} of {len(spec.order)}")
        self._join_runs = frozenset(int(r) for r in spec.join_runs)
        if self._join_runs and (self.join is None or not all(0 <= r < len(spec.order) for r in self._join_runs)):
            raise ValueError(f"the stream cannot be joined before the runs {sorted(self._join_runs)} of {len(spec.order)}")

    # ------------------------------------------------------------------ weights
    def tensor_needs(self) -> dict[str, TensorNeed]:
        return tensor_needs_of(self.spec)

    def parts(self):
        yield self.embedding
        for b in self.blocks:
            yield from b.parts()
        if self.join is not None:
            yield self.join
        yield self.final_norm
        yield self.head

    def all_parts(self):
        """Every part, those inside other parts (`inner_parts()`, loaded by their owners) included."""
        for part in self.parts():
            yield part
            yield from getattr(part, "inner_parts", lambda: [])()

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        """`tensors`: checked, converted, on the device (see weights.loader)."""
        for part in self.parts():
            part.load(tensors)
        if getattr(self.head, "tied", False):
            self.head.tie(self.embedding.weight)
        self.loaded = True

    # ------------------------------------------------------------------ cache
    def cache_needs(self) -> list:
        """Per layer: the mixer's KVCacheNeed, StateNeed or None; for a block whose other
        parts keep state too (`cache_holders()`), a tuple with every holder's need. After the
        layers: one need for every part outside them that keeps something per request."""
        out = []
        for layer in self._unit_layer:
            b = self.blocks[layer]
            holders = getattr(b, "cache_holders", None)
            out.append(tuple(h.cache_need() for h in holders()) if holders is not None else b.mixer.cache_need())
        return out + [part.cache_need() for part in self._own_holders]

    def cache_holder(self, key):
        """The part behind a cache manager's holder key: a layer's mixer, or for the key
        (layer, place) that place among the block's cache holders."""
        if isinstance(key, tuple):
            return self.blocks[self._unit_layer[key[0]]].cache_holders()[key[1]]
        if key >= len(self._unit_layer):
            return self._own_holders[key - len(self._unit_layer)]
        return self.blocks[self._unit_layer[key]].mixer

    def cache_sources(self) -> list[int | None]:
        """Per layer: the layer whose cache it reads instead of its own, or None."""
        sources = [getattr(b.mixer, "cache_from", None) for b in self.blocks]
        needs = self.cache_needs()
        for layer, src in enumerate(sources):
            if src is None:
                continue
            if not 0 <= src < len(self.blocks) or needs[src] is None or sources[src] is not None or (
                    isinstance(needs[src], tuple) and needs[src][0] is None):
                raise ValueError(f"layer {layer} reads the cache of layer {src}, which keeps none of its own")
            # The reader must see the cache as its owner keeps it: the same heads and head
            # size, and no further back than the owner's window (pages behind that window
            # are given back while the request runs).
            reads = getattr(self.blocks[layer].mixer, "cache_read_need", None)
            want, have = (reads() if reads is not None else None), needs[src]
            if isinstance(have, tuple):
                have = have[0]  # (a block's cache holders start with its mixer)
            if want is not None and hasattr(have, "n_kv_heads"):
                if (want.n_kv_heads, want.head_dim) != (have.n_kv_heads, have.head_dim):
                    raise ValueError(
                        f"layer {layer} reads the cache of layer {src} as {want.n_kv_heads} kv heads of size "
                        f"{want.head_dim}, but it holds {have.n_kv_heads} of size {have.head_dim}")
                if have.window is not None and want.window is not None and want.keep_first > have.keep_first:
                    raise ValueError(f"layer {layer} reads the first {want.keep_first} tokens of layer {src}'s cache, which "
                                     f"keeps {have.keep_first} only")
                if have.window is not None and (want.window is None or want.window > have.window):
                    raise ValueError(
                        f"layer {layer} reads {'every key' if want.window is None else f'a window of {want.window}'} "
                        f"of layer {src}'s cache, which keeps a window of {have.window} only")
        return sources

    def planners(self) -> list:
        """The parts that plan steps on the host, one per distinct plan_key()."""
        seen: dict = {}
        for part in self.all_parts():
            key_of = getattr(part, "plan_key", None)
            key = key_of() if key_of is not None else None
            if key is not None and key not in seen:
                seen[key] = part
        return list(seen.items())

    def _bind_block(self, b, mine) -> None:
        if hasattr(b, "cache_holders"):
            for holder, binding in zip(b.cache_holders(), mine):
                if binding is not None:
                    holder.bind_cache(binding)
        elif mine is not None:
            b.mixer.bind_cache(mine[0] if isinstance(mine, list) else mine)

    def bind_caches(self, bindings: list) -> None:
        for place, part in enumerate(self._own_holders):
            part.bind_cache(bindings[len(self._unit_layer) + place])
        if self.spec.cache_per_run:
            # One binding per run: a block is pointed at its run's cache right before it runs
            # (`forward`); here each block gets the binding of its first run, so that whatever the
            # parts derive from a binding (page size, kernels' shapes) is known before a step.
            if any(getattr(b.mixer, "cache_from", None) is not None for b in self.blocks):
                raise ValueError("a model that keeps a cache per run cannot have layers that read another's cache")
            self._run_bindings = list(bindings[: len(self._unit_layer)])
            seen = set()
            for run, layer in enumerate(self.spec.order):
                if layer not in seen:
                    seen.add(layer)
                    self._bind_block(self.blocks[layer], bindings[run])
            return
        sources = self.cache_sources()
        for layer, b in enumerate(self.blocks):
            src = sources[layer] if sources[layer] is not None else layer
            if hasattr(b, "cache_holders"):
                mine = list(bindings[layer])
                if src != layer:
                    theirs = bindings[src]
                    mine[0] = theirs[0] if isinstance(theirs, list) else theirs
                for holder, binding in zip(b.cache_holders(), mine):
                    if binding is not None:
                        holder.bind_cache(binding)
            elif bindings[src] is not None:
                theirs = bindings[src]
                b.mixer.bind_cache(theirs[0] if isinstance(theirs, list) else theirs)

    @staticmethod
    def _rejoin_stream(x, delta, entered):
        """The embedding's output enters the stream again: with the pending output where its kind
        can carry a row of its own (the next norm's kernel then adds it in the same pass), else now."""
        if delta is not None and hasattr(delta, "with_also"):
            return x, delta.with_also(entered)
        x.add_(entered)
        return x, delta

    # ------------------------------------------------------------------ forward
    def forward(self, batch: StepBatch) -> torch.Tensor | None:
        """Runs the batch's tokens through every layer in order; returns fp32 logits
        [R, vocab] at `batch.want_rows`, or None when none are wanted."""
        if not self.loaded:
            raise RuntimeError("the model has no weights loaded")
        x = self.embedding.forward(batch.tokens, batch)
        delta = None
        entered = x.clone() if self._rejoin or self._join_runs else None  # (the stream is updated in place)
        repeated = self._run_bindings is not None and len(self.spec.order) != len(set(self.spec.order))
        for run, index in enumerate(self.spec.order):
            block = self.blocks[index]
            if repeated:
                self._bind_block(block, self._run_bindings[run])
            if run in self._rejoin:
                x, delta = self._rejoin_stream(x, delta, entered)
            if run in self._join_runs:
                x, delta = self.join.forward(x, delta, entered), None
            x, delta = block.forward(x, delta, batch)
        if batch.want_rows is None or batch.want_rows.numel() == 0:
            return None
        h = self.final_norm.forward(x, delta, rows=batch.want_rows)
        return self.head.forward(h)
