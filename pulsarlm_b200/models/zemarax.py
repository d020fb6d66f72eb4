"""The Zemarax decoder, described as data and registered by name.

A layer: x += norm1b(mixer(norm1(x))), then, where the layer has a feed-forward, x += norm2b(ff(norm2(x))), all four RMS
norms with weights around zero (the "sandwich_norm" block). Tensor names: `embed`, `bigram`, `pos`, `final.norm`, `head`,
and per layer `l<i>.`: norm1, norm1b, norm2, norm2b, mix.{q, k, v, q.norm, k.norm, sink, o} (attention), mix.{q, k, v, g,
i, i.b, f, f.b, norm, o} (mlstm), mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, sink, o} (latent_attention), mlp.{gate, up,
down} or mlp.{router, router.b, e<j>.up, e<j>.down, shared.up, shared.down, shared.sg}.
"""

from __future__ import annotations

from ..config.registry import register_architecture
from ..config.zemarax import ZemaraxConfig, ZemaraxLayer
from ..parts.spec import LayerSpec, ModelSpec, PartSpec


def _mixer(layer: ZemaraxLayer, width: int, eps: float, m: str) -> PartSpec:
    x = layer.mixer
    params = {"hidden_size": width, "n_heads": x.heads, "head_dim": x.dim, "value_dim": x.vdim}

    def names(**roles: str) -> dict:
        return {role: m + name for role, name in roles.items()}

    if layer.type == "attention":
        params.update(n_kv_heads=x.kv_heads, scale=x.scale, window=x.window, keep_first=x.keep_first, qk_norm="per_head",
                      norm_eps=eps, split_weights=False, position=PartSpec("none"))
        return PartSpec("normed_attention", params, names(q="q", k="k", v="v", q_norm="q.norm", k_norm="k.norm",
                                                          sink="sink", o="o"))
    if layer.type == "mlstm":
        params.update(gate_cap=x.gate_cap, eps=eps)
        return PartSpec("matrix_memory", params, names(q="q", k="k", v="v", g="g", i="i", i_bias="i.b", f="f",
                                                       f_bias="f.b", norm="norm", o="o"))
    params.update(query_rank=x.q_rank, latent_rank=x.kv_rank, scale=x.scale, eps=eps, sink=True, cache_from=x.kv_from,
                  split_weights=False)
    return PartSpec("latent_attention", params, names(query_down="dq", query_norm="dq.norm", q="uq", down="dkv",
                                                      latent_norm="dkv.norm", up_k="uk", up_v="uv", sink="sink", o="o"))


def _feed_forward(layer: ZemaraxLayer, width: int, f: str) -> PartSpec | None:
    mlp = layer.mlp
    if mlp is None:
        return None
    if mlp.kind == "dense":
        return PartSpec("gated_mlp", {"hidden_size": width, "intermediate_size": mlp.ff},
                        {"gate": f + "gate", "up": f + "up", "down": f + "down"})
    names = {"router": f + "router", "logit_bias": f + "router.b", "expert_up": f + "e{e}.up", "expert_down": f + "e{e}.down"}
    if mlp.shared_ff is not None:
        names.update(shared_up=f + "shared.up", shared_down=f + "shared.down", shared_gate_row=f + "shared.sg")
    return PartSpec("moe", {"hidden_size": width, "expert_size": mlp.ff, "n_experts": mlp.experts, "top": mlp.top,
                            "shared_size": mlp.shared_ff, "expert": "gelu"}, names)


def describe_zemarax(cfg: ZemaraxConfig) -> ModelSpec:
    width, eps = cfg.width, cfg.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"hidden_size": width, "eps": eps, "unit_offset": True}, {"weight": name})

    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        norms = {"mixer": norm(p + "norm1"), "mixer_out": norm(p + "norm1b")}
        extras = {}
        if layer.mlp is not None:
            norms.update(feed_forward=norm(p + "norm2"), feed_forward_out=norm(p + "norm2b"))
        else:
            # (a layer without feed-forward may still store its norms)
            extras["ignored"] = {p + "norm2": (width,), p + "norm2b": (width,)}
        layers.append(LayerSpec("sandwich_norm", _mixer(layer, width, eps, p + "mix."),
                                _feed_forward(layer, width, p + "mlp."), norms, extras))
    sizes = {"vocab_size": cfg.vocab, "hidden_size": width}
    return ModelSpec(
        hidden_size=width,
        vocab_size=cfg.vocab,
        embedding=PartSpec("pair_hash_table",
                           {**sizes, "buckets": cfg.pairs.buckets, "mul_prev": cfg.pairs.mul_prev,
                            "mul_cur": cfg.pairs.mul_cur, "scale": cfg.embedding_scale, "positions": cfg.max_positions},
                           {"weight": "embed", "pairs": "bigram", "places": "pos"}),
        layers=layers,
        order=list(range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear", {**sizes, "scale": cfg.logit_scale}, {"weight": "head"}),
        max_positions=cfg.max_positions,
    )


register_architecture("Zemarax", ZemaraxConfig.from_text, describe_zemarax, model_types=("zemarax",), replace=True)
