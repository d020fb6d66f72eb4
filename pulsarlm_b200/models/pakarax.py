"""The Pakarax decoder, described as data and registered by name.

A layer: h = norm1(x), x += (norm(left(h)) + norm(right(h))) / 2 + ff(h) (the "parallel" block with one norm and a
side-by-side mixer). A run of layers may repeat with the same weights; every pass has a cache and states of its own, and
before every pass x <- W [x; x0], x0 the embedding's output. Tensor names: `embed`, `loop.in`, `final.norm`, `head`, and
per layer `l<i>.` + norm1, mix.left.*, mix.right.*, mlp.*.
"""

from __future__ import annotations

from ..config.pakarax import PakaraxConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec

SLOPE_OCTAVES = 8.0   # head h of H is marked down 2^(-8 (h + 1) / H) per token of distance
DECAY_SCALE = 8.0     # log a = -8 r softplus(lambda)


def _feed_forward(m, width: int, f: str) -> PartSpec | None:
    if m is None:
        return None
    if m.kind == "dense":
        return PartSpec("gated_mlp", {"hidden_size": width, "intermediate_size": m.ff, "activation": "clamped",
                                      "limit": m.limit}, {n: f + n for n in ("gate", "up", "down")})
    tensors = {"router": f + "router", "expert_gate": f + "e{e}.gate", "expert_up": f + "e{e}.up",
               "expert_down": f + "e{e}.down"}
    if m.shared_ff is not None:
        tensors.update(shared_gate=f + "shared.gate", shared_up=f + "shared.up", shared_down=f + "shared.down",
                       shared_gate_row=f + "shared.sg")
    return PartSpec("moe", {"hidden_size": width, "expert_size": m.ff, "n_experts": m.experts, "top": m.top,
                            "shared_size": m.shared_ff, "scores": "sigmoid", "renormalise": False, "expert": "clamped",
                            "expert_limit": m.limit, "shared_limit": m.shared_limit, "weigh_input": True}, tensors)


def describe_pakarax(cfg: PakaraxConfig) -> ModelSpec:
    width = cfg.width

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"hidden_size": width, "eps": cfg.norm_eps}, {"weight": name})

    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        a, r = layer.left, layer.right
        left, right = p + "mix.left.", p + "mix.right."
        attention = PartSpec(
            "filtered_attention",
            {"hidden_size": width, "n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "value_dim": a.vdim,
             "taps": a.taps, "scale": a.scale, "slope_octaves": SLOPE_OCTAVES, "split_weights": False,
             "temperature": (a.temp_coef, a.temp_every) if a.temp_coef is not None else None},
            {**{n: left + n for n in ("q", "k", "v", "o", "sink")},
             **{n + "_bias": left + n + ".b" for n in ("q", "k", "v", "o")},
             **{n + "_conv": left + n + ".conv" for n in ("q", "k", "v")}})
        recurrence = PartSpec(
            "linear_recurrence",
            {"hidden_size": width, "width": r.width, "blocks": r.blocks, "taps": r.taps, "decay_scale": DECAY_SCALE},
            {**{n: right + n for n in ("y", "x", "conv", "ra", "ri", "lam", "o")},
             **{n + "_bias": right + n + ".b" for n in ("y", "x", "conv", "ra", "ri")}})
        mixer = PartSpec("side_by_side", {"hidden_size": width, "eps": cfg.norm_eps, "left": attention,
                                          "right": recurrence},
                         {"left_norm": left + "out", "right_norm": right + "out"})
        layers.append(LayerSpec(block="parallel", mixer=mixer, feed_forward=_feed_forward(layer.mlp, width, p + "mlp."),
                                norms={"mixer": norm(p + "norm1")}))
    order, begins = cfg.runs()
    sizes = {"vocab_size": cfg.vocab, "hidden_size": width}
    return ModelSpec(
        hidden_size=width,
        vocab_size=cfg.vocab,
        embedding=PartSpec("table", dict(sizes), {"weight": "embed"}),
        layers=layers,
        order=order,
        final_norm=norm("final.norm"),
        head=PartSpec("linear", {**sizes, "scale": cfg.logit_scale, "softcap": cfg.logit_softcap}, {"weight": "head"}),
        cache_per_run=True,
        join=PartSpec("concat_linear", {"hidden_size": width}, {"weight": "loop.in"}) if cfg.loop is not None else None,
        join_runs=tuple(begins),
    )


register_architecture("Pakarax", PakaraxConfig.from_text, describe_pakarax, model_types=("pakarax",), replace=True)
