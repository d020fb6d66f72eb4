"""ZemaraxConfig: the typed configuration of the Zemarax decoder.

Zemarax lists its layers one by one. Every sublayer is normed before and after (RMS norms whose weights are stored around
zero). Mixers:

* `attention`: grouped-query attention with an RMS norm on every head of q and k, no rotation, a sliding window beside
  which a sequence's first tokens stay in reach, a learned sink per head, key and value sizes of their own;
* `mlstm`: a matrix memory with exponential gates (state, normaliser and stabiliser per head);
* `latent_attention`: attention over a cached latent, the queries through a latent of their own, a learned sink per head;
  a layer with `kv_from` reads the latents of an earlier such layer instead of making any.

Feed-forward: a gated one with SiLU, or routed experts with GELU (biased logits, weights by the softmax over the chosen
ones) beside a shared expert with a gate per token, or none. The embedding is scaled and adds a row of a second table
chosen by a hash of (token before, token) and a learned vector per position; the head has its own table, its logits scaled.
"""

from __future__ import annotations

import dataclasses

from .base import ConfigError, read_field, require_positive

MIXERS = ("attention", "mlstm", "latent_attention")


@dataclasses.dataclass(frozen=True)
class ZemaraxMixer:
    """`mixer` of a layer, whatever its type; what a type does not have stays at its default."""

    heads: int
    dim: int
    vdim: int
    scale: float | None = None        # attention, latent_attention
    kv_heads: int | None = None       # attention
    window: int | None = None         # attention (None: every earlier token)
    keep_first: int = 0
    gate_cap: float | None = None     # mlstm
    q_rank: int | None = None         # latent_attention
    kv_rank: int | None = None
    kv_from: int | None = None


@dataclasses.dataclass(frozen=True)
class ZemaraxFeedForward:
    """`mlp` of a layer. kind "dense": `ff`. kind "moe": an expert's `ff`; `experts`, `top`; the shared expert's
    `shared_ff` (None: none)."""

    kind: str
    ff: int
    experts: int = 0
    top: int = 0
    shared_ff: int | None = None


@dataclasses.dataclass(frozen=True)
class ZemaraxLayer:
    type: str
    mixer: ZemaraxMixer
    mlp: ZemaraxFeedForward | None


@dataclasses.dataclass(frozen=True)
class PairTable:
    """`embedding.bigram`: rows of the second table and the hash's two multipliers."""

    buckets: int
    mul_prev: int
    mul_cur: int


@dataclasses.dataclass(frozen=True)
class ZemaraxConfig:
    architecture: str
    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    embedding_scale: float
    pairs: PairTable
    layers: tuple[ZemaraxLayer, ...]
    logit_scale: float = 1.0

    @staticmethod
    def from_text(text: dict) -> "ZemaraxConfig":
        entries = read_field(text, "layers", list)
        if not entries:
            raise ConfigError("config.json: 'layers' must list at least one layer")
        layers: list[ZemaraxLayer] = []
        for i, entry in enumerate(entries):
            layers.append(_read_layer(entry, i, layers))
        embedding = read_field(text, "embedding", dict)
        bigram = read_field(embedding, "bigram", dict)
        cfg = ZemaraxConfig(
            architecture=str(text.get("architecture") or "Zemarax"),
            vocab=read_field(text, "vocab", int),
            width=read_field(text, "width", int),
            max_positions=read_field(text, "max_positions", int),
            norm_eps=read_field(read_field(text, "norm", dict), "eps", float),
            embedding_scale=read_field(embedding, "scale", float, 1.0),
            pairs=PairTable(*(read_field(bigram, name, int) for name in ("buckets", "mul_prev", "mul_cur"))),
            layers=tuple(layers),
            logit_scale=read_field(text, "logit_scale", float, 1.0),
        )
        for name, value in (("vocab", cfg.vocab), ("width", cfg.width), ("max_positions", cfg.max_positions),
                            ("embedding.bigram.buckets", cfg.pairs.buckets)):
            require_positive(name, value)
        return cfg

    def to_text(self) -> dict:
        """A config.json that `from_text` reads back to an equal configuration."""
        layers = []
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            mixer = {name: value for name, value in dataclasses.asdict(m).items()
                     if value is not None and name not in ("window", "keep_first")}
            if m.window is not None:
                mixer["mask"] = {"size": m.window, "keep_first": m.keep_first}
            mlp = None
            if f is not None and f.kind == "dense":
                mlp = {"kind": "dense", "ff": f.ff}
            elif f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
                if f.shared_ff is not None:
                    mlp["shared"] = {"ff": f.shared_ff}
            layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "max_positions": self.max_positions, "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale,
                "embedding": {"scale": self.embedding_scale, "bigram": dataclasses.asdict(self.pairs)}, "layers": layers}


def _read_layer(entry, i: int, before: list[ZemaraxLayer]) -> ZemaraxLayer:
    where = f"layers[{i}]"
    if not isinstance(entry, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    kind = read_field(entry, "type", str)
    if kind not in MIXERS:
        raise ConfigError(f"config.json: {where}.type {kind!r} is unknown (known: {', '.join(MIXERS)})")
    mixer = read_field(entry, "mixer", dict)
    heads, dim = read_field(mixer, "heads", int), read_field(mixer, "dim", int)
    sizes = {"heads": heads, "dim": dim, "vdim": read_field(mixer, "vdim", int, dim)}
    extra: dict = {}
    if kind == "attention":
        sizes["kv_heads"] = read_field(mixer, "kv_heads", int, heads)
        extra["scale"] = read_field(mixer, "scale", float)
        if mixer.get("mask") is not None:
            mask = read_field(mixer, "mask", dict)
            extra["window"] = read_field(mask, "size", int)
            extra["keep_first"] = read_field(mask, "keep_first", int, 0)
            require_positive(f"{where}.mixer.mask.size", extra["window"])
            if extra["keep_first"] < 0:
                raise ConfigError(f"config.json: {where}.mixer.mask.keep_first must not be negative")
    elif kind == "mlstm":
        extra["gate_cap"] = read_field(mixer, "gate_cap", float)
        if extra["gate_cap"] <= 0.0:
            raise ConfigError(f"config.json: {where}.mixer.gate_cap must be positive, got {extra['gate_cap']}")
    else:
        sizes["q_rank"], sizes["kv_rank"] = read_field(mixer, "q_rank", int), read_field(mixer, "kv_rank", int)
        extra["scale"] = read_field(mixer, "scale", float)
        extra["kv_from"] = source = read_field(mixer, "kv_from", int, None)
        if source is not None:
            if not 0 <= source < i or before[source].type != kind or before[source].mixer.kv_from is not None:
                raise ConfigError(f"config.json: {where}.mixer.kv_from {source} is no earlier latent layer that makes its own "
                                  f"latents")
            if before[source].mixer.kv_rank != sizes["kv_rank"]:
                raise ConfigError(f"config.json: {where} reads latents of {sizes['kv_rank']} from layer {source}, which makes "
                                  f"latents of {before[source].mixer.kv_rank}")
    for name, value in sizes.items():
        require_positive(f"{where}.mixer.{name}", value)
    if heads % sizes.get("kv_heads", 1):
        raise ConfigError(f"config.json: {where}.mixer: {heads} heads are not a multiple of {sizes['kv_heads']} kv_heads")
    return ZemaraxLayer(kind, ZemaraxMixer(**sizes, **extra), _read_mlp(entry.get("mlp"), where))


def _read_mlp(mlp, where: str) -> ZemaraxFeedForward | None:
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"config.json: {where}.mlp must be an object or null")
    kind = read_field(mlp, "kind", str)
    if kind == "dense":
        out = ZemaraxFeedForward("dense", read_field(mlp, "ff", int))
    elif kind == "moe":
        router = read_field(mlp, "router", dict)
        shared = read_field(mlp, "shared", dict) if mlp.get("shared") is not None else None
        out = ZemaraxFeedForward("moe", read_field(read_field(mlp, "expert", dict), "ff", int),
                                 read_field(router, "experts", int), read_field(router, "top", int),
                                 read_field(shared, "ff", int) if shared is not None else None)
        for name, value in (("router.experts", out.experts), ("router.top", out.top)):
            require_positive(f"{where}.mlp.{name}", value)
        if out.top > out.experts:
            raise ConfigError(f"config.json: {where}.mlp.router: {out.top} of {out.experts} experts cannot be chosen")
        if out.shared_ff is not None:
            require_positive(f"{where}.mlp.shared.ff", out.shared_ff)
    else:
        raise ConfigError(f"config.json: {where}.mlp.kind {kind!r} is unknown (known: dense, moe)")
    require_positive(f"{where}.mlp ff", out.ff)
    return out
