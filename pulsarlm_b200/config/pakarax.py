"""PakaraxConfig: the typed configuration of the Pakarax decoder.

Pakarax lists its layers one by one. A layer has one RMS norm; its mixer and its feed-forward read
the norm's output and enter the residual stream together. The mixer is two side by side:
grouped-query attention over queries, keys and values that pass a short convolution each (biased
projections, a temperature on the queries, a linear bias by distance, a learned sink per head) and
a gated linear recurrence behind a short convolution beside a GELU branch; the two outputs are
normed and averaged. The feed-forward is a gated one with a clamped unit, or routed experts of the
same form (sigmoid scores that weigh the experts' inputs) beside a shared expert with a gate per
token, or absent. A run of layers may be repeated with the same weights (`loop`), every pass with a
cache and state of its own; before every pass, the first one too, the stream is made anew from
itself and the embedding's output by one projection. Logits are scaled and capped.
"""

from __future__ import annotations

import dataclasses

from .base import ConfigError, read_field, require_positive

MIXERS = ("parallel",)


@dataclasses.dataclass(frozen=True)
class PakaraxAttention:
    """`mixer.left`."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    scale: float
    temp_coef: float | None = None    # None: the queries are not scaled by position
    temp_every: int | None = None


@dataclasses.dataclass(frozen=True)
class PakaraxRecurrence:
    """`mixer.right`."""

    width: int
    blocks: int
    taps: int


@dataclasses.dataclass(frozen=True)
class PakaraxFeedForward:
    """`mlp` of a layer. kind "dense": `ff`, `limit`. kind "moe": an expert's `ff` and `limit`; `experts`, `top`;
    the shared expert's `shared_ff` and `shared_limit` (None: none)."""

    kind: str
    ff: int
    limit: float
    experts: int = 0
    top: int = 0
    shared_ff: int | None = None
    shared_limit: float | None = None


@dataclasses.dataclass(frozen=True)
class PakaraxLayer:
    """One entry of config.json's `layers`."""

    type: str
    left: PakaraxAttention
    right: PakaraxRecurrence
    mlp: PakaraxFeedForward | None


@dataclasses.dataclass(frozen=True)
class PakaraxConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[PakaraxLayer, ...]
    logit_scale: float = 1.0
    logit_softcap: float | None = None
    loop: tuple[int, int, int] | None = None   # (start, stop, times)

    def runs(self) -> tuple[list[int], list[int]]:
        """(the layers in the order they run, the places in that order where a pass begins)."""
        start, stop, times = self.loop or (0, 0, 0)
        order, begins = list(range(start)), []
        for _ in range(times if stop > start else 0):
            begins.append(len(order))
            order += range(start, stop)
        return order + list(range(stop, len(self.layers))), begins

    @staticmethod
    def from_text(text: dict) -> "PakaraxConfig":
        entries = read_field(text, "layers", list)
        if not entries:
            raise ConfigError("config.json: 'layers' must list at least one layer")
        loop = None
        if text.get("loop") is not None:
            given = read_field(text, "loop", dict)
            loop = tuple(read_field(given, name, int) for name in ("start", "stop", "times"))
            if not 0 <= loop[0] <= loop[1] <= len(entries) or loop[2] < 1:
                raise ConfigError(f"config.json: loop start {loop[0]}, stop {loop[1]}, times {loop[2]} do not fit "
                                  f"{len(entries)} layers")
        cfg = PakaraxConfig(
            architecture=str(text.get("architecture") or "Pakarax"),
            vocab=read_field(text, "vocab", int),
            width=read_field(text, "width", int),
            norm_eps=read_field(read_field(text, "norm", dict), "eps", float),
            layers=tuple(_read_layer(entry, f"layers[{i}]") for i, entry in enumerate(entries)),
            logit_scale=read_field(text, "logit_scale", float, 1.0),
            logit_softcap=read_field(text, "logit_softcap", float, None),
            loop=loop,
        )
        require_positive("vocab", cfg.vocab)
        require_positive("width", cfg.width)
        if cfg.logit_softcap is not None:
            require_positive("logit_softcap", cfg.logit_softcap)
        return cfg

    def to_text(self) -> dict:
        """A config.json that `from_text` reads back to an equal configuration."""
        layers = []
        for layer in self.layers:
            a, r, m = layer.left, layer.right, layer.mlp
            left: dict = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "conv": a.taps,
                          "scale": a.scale}
            if a.temp_coef is not None:
                left["q_temp"] = {"coef": a.temp_coef, "every": a.temp_every}
            mlp = None
            if m is not None and m.kind == "dense":
                mlp = {"kind": "dense", "ff": m.ff, "limit": m.limit}
            elif m is not None:
                mlp = {"kind": "moe", "expert": {"ff": m.ff, "limit": m.limit},
                       "router": {"experts": m.experts, "top": m.top}}
                if m.shared_ff is not None:
                    mlp["shared"] = {"ff": m.shared_ff, "limit": m.shared_limit}
            layers.append({"type": layer.type, "mixer": {"left": left, "right": {"width": r.width, "blocks": r.blocks,
                                                                                 "conv": r.taps}}, "mlp": mlp})
        out: dict = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                     "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale, "layers": layers}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out


def _read_layer(entry, where: str) -> PakaraxLayer:
    if not isinstance(entry, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    kind = read_field(entry, "type", str)
    if kind not in MIXERS:
        raise ConfigError(f"config.json: {where}.type {kind!r} is unknown (known: {', '.join(MIXERS)})")
    mixer = read_field(entry, "mixer", dict)
    left, right = read_field(mixer, "left", dict), read_field(mixer, "right", dict)
    heads, dim = read_field(left, "heads", int), read_field(left, "dim", int)
    coef = every = None
    if left.get("q_temp") is not None:
        temp = read_field(left, "q_temp", dict)
        coef, every = read_field(temp, "coef", float), read_field(temp, "every", int)
        require_positive(f"{where}.mixer.left.q_temp.every", every)
    attention = PakaraxAttention(
        heads=heads, kv_heads=read_field(left, "kv_heads", int, heads), dim=dim, vdim=read_field(left, "vdim", int, dim),
        taps=read_field(left, "conv", int), scale=read_field(left, "scale", float), temp_coef=coef, temp_every=every)
    recurrence = PakaraxRecurrence(width=read_field(right, "width", int), blocks=read_field(right, "blocks", int),
                                   taps=read_field(right, "conv", int))
    for name, value in (("left.heads", attention.heads), ("left.kv_heads", attention.kv_heads), ("left.dim", dim),
                        ("left.vdim", attention.vdim), ("left.conv", attention.taps), ("right.width", recurrence.width),
                        ("right.blocks", recurrence.blocks), ("right.conv", recurrence.taps)):
        require_positive(f"{where}.mixer.{name}", value)
    if attention.heads % attention.kv_heads:
        raise ConfigError(f"config.json: {where}.mixer.left: {attention.heads} heads are not a multiple of "
                          f"{attention.kv_heads} kv_heads")
    if recurrence.width % recurrence.blocks:
        raise ConfigError(f"config.json: {where}.mixer.right: width {recurrence.width} does not split into "
                          f"{recurrence.blocks} blocks")
    return PakaraxLayer(kind, attention, recurrence, _read_mlp(entry.get("mlp"), where))


def _read_mlp(mlp, where: str) -> PakaraxFeedForward | None:
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"config.json: {where}.mlp must be an object or null")
    kind = read_field(mlp, "kind", str)
    if kind == "dense":
        out = PakaraxFeedForward("dense", read_field(mlp, "ff", int), read_field(mlp, "limit", float))
    elif kind == "moe":
        expert, router = read_field(mlp, "expert", dict), read_field(mlp, "router", dict)
        shared = read_field(mlp, "shared", dict) if mlp.get("shared") is not None else None
        out = PakaraxFeedForward(
            "moe", read_field(expert, "ff", int), read_field(expert, "limit", float), read_field(router, "experts", int),
            read_field(router, "top", int), read_field(shared, "ff", int) if shared is not None else None,
            read_field(shared, "limit", float) if shared is not None else None)
        for name, value in (("router.experts", out.experts), ("router.top", out.top)):
            require_positive(f"{where}.mlp.{name}", value)
        if out.top > out.experts:
            raise ConfigError(f"config.json: {where}.mlp.router: {out.top} of {out.experts} experts cannot be chosen")
        if shared is not None:
            require_positive(f"{where}.mlp.shared.ff", out.shared_ff)
    else:
        raise ConfigError(f"config.json: {where}.mlp.kind {kind!r} is unknown (known: dense, moe)")
    require_positive(f"{where}.mlp ff", out.ff)
    return out
