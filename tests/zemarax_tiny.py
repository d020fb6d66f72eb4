"""Small Zemarax configurations and random weights for the tests.

The configurations differ from each other in every size and constant: layer order (each mixer first somewhere), widths,
head counts (query heads per kv head 1, 2, 3 and 4), key sizes above and below the value size, windows and kept first
tokens (within a page, over a page's edge, more than the window, none; also no window), latent ranks with and without
a tensor-core kernel, query latents of other sizes, layers that read an earlier layer's latents with other heads and
value sizes, matrix memories with and without a chunked kernel, gate caps that bite, dense and routed feed-forwards (with
and without a shared expert, one chosen expert and all), a layer without feed-forward, embedding and logit scales (also
1). Weights are drawn with torch and written with the `safetensors` package, so the engine's reader and its names are
checked against an independent file.
"""

from __future__ import annotations

import json
import os
import tempfile

import torch

import plain_zemarax


def dense(ff):
    return {"kind": "dense", "ff": ff}


def routed(ff, experts, top, shared=None):
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared}
    return mlp


def windowed(heads, kv_heads, dim, vdim, mlp, size=None, keep_first=0, scale=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
             "scale": scale if scale is not None else 1.5 * dim ** -0.5}
    if size is not None:
        mixer["mask"] = {"size": size, "keep_first": keep_first}
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def memory(heads, dim, vdim, mlp, cap=15.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def latent(heads, dim, vdim, q_rank, kv_rank, mlp, kv_from=None, scale=None):
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
             "scale": scale if scale is not None else 1.5 * dim ** -0.5}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def config(vocab, width, eps, scales, pairs, layers, positions=1024):
    """scales: (embedding scale, logit scale); pairs: (buckets, mul_prev, mul_cur)."""
    return {"architecture": "Zemarax", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": eps},
            "embedding": {"scale": scales[0], "bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), pairs))},
            "logit_scale": scales[1], "layers": layers}


CONFIG_A = config(211, 72, 1e-5, (6.0, 1.5), (97, 31, 5), [
    windowed(4, 2, 16, 24, routed(24, 8, 3, 40), size=21, keep_first=3),
    memory(3, 16, 24, dense(96)),
    latent(4, 24, 16, 40, 32, None),
    memory(2, 32, 8, routed(16, 5, 1), cap=2.0),
    latent(3, 8, 24, 24, 32, dense(60), kv_from=2),
])
CONFIG_B = config(97, 40, 1e-6, (1.0, 1.0), (13, 3, 11), [
    latent(2, 12, 8, 20, 24, dense(56), scale=0.9),
    memory(5, 6, 10, None, cap=4.5),
    windowed(3, 3, 8, 16, routed(16, 6, 6), size=9, keep_first=20, scale=0.5),
    windowed(4, 1, 20, 12, dense(24)),
    latent(4, 6, 20, 12, 24, routed(12, 4, 2, 20), kv_from=0, scale=0.7),
])
CONFIG_C = config(128, 64, 1e-6, (3.0, 0.7), (251, 1, 2), [
    memory(2, 64, 128, dense(80), cap=9.0),
    windowed(8, 2, 64, 32, dense(48), size=40, keep_first=17, scale=0.2),
    latent(8, 32, 48, 64, 64, routed(32, 8, 2, 48)),
    windowed(2, 1, 64, 64, dense(80), size=70, keep_first=64, scale=0.25),
    memory(4, 48, 80, routed(24, 4, 3)),
    windowed(3, 1, 128, 96, dense(40), size=33, keep_first=5, scale=0.15),
])
CONFIGS = {"A": (CONFIG_A, 16), "B": (CONFIG_B, 32), "C": (CONFIG_C, 16)}


def tensor_shapes(cfg: dict) -> dict[str, tuple[int, ...]]:
    w = cfg["width"]
    shapes = {"embed": (cfg["vocab"], w), "head": (cfg["vocab"], w), "pos": (cfg["max_positions"], w),
              "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, w), "final.norm": (w,)}
    for i, layer in enumerate(cfg["layers"]):
        p, x, m = f"l{i}.", f"l{i}.mix.", layer["mixer"]
        heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
        shapes[p + "norm1"] = shapes[p + "norm1b"] = (w,)
        shapes[x + "o"] = (w, heads * vdim)
        if layer["type"] == "attention":
            kv = m["kv_heads"]
            shapes.update({x + "q": (heads * dim, w), x + "k": (kv * dim, w), x + "v": (kv * vdim, w), x + "q.norm": (dim,),
                           x + "k.norm": (dim,), x + "sink": (heads,)})
        elif layer["type"] == "mlstm":
            shapes.update({x + "q": (heads * dim, w), x + "k": (heads * dim, w), x + "v": (heads * vdim, w),
                           x + "g": (heads * vdim, w), x + "i": (heads, w), x + "i.b": (heads,), x + "f": (heads, w),
                           x + "f.b": (heads,), x + "norm": (heads * vdim,)})
        else:
            rank = m["kv_rank"]
            shapes.update({x + "dq": (m["q_rank"], w), x + "dq.norm": (m["q_rank"],), x + "uq": (heads * dim, m["q_rank"]),
                           x + "uk": (heads * dim, rank), x + "uv": (heads * vdim, rank), x + "sink": (heads,)})
            if m.get("kv_from") is None:
                shapes.update({x + "dkv": (rank, w), x + "dkv.norm": (rank,)})
        mlp = layer["mlp"]
        if mlp is None:
            continue
        shapes[p + "norm2"] = shapes[p + "norm2b"] = (w,)
        f = p + "mlp."
        if mlp["kind"] == "dense":
            shapes.update({f + "gate": (mlp["ff"], w), f + "up": (mlp["ff"], w), f + "down": (w, mlp["ff"])})
        else:
            experts, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
            for e in range(experts):
                shapes[f + f"e{e}.up"], shapes[f + f"e{e}.down"] = (ff, w), (w, ff)
            shapes[f + "router"], shapes[f + "router.b"] = (experts, w), (experts,)
            if mlp.get("shared"):
                fs = mlp["shared"]["ff"]
                shapes.update({f + "shared.up": (fs, w), f + "shared.down": (w, fs), f + "shared.sg": (1, w)})
    return shapes


def random_weights(cfg: dict, seed: int, dtype: torch.dtype = torch.float32, sharp: float = 1.0) -> dict:
    """Matrices N(0, 1/sqrt(in)); plain norm weights 1 + 0.2 N (a q.norm times `sharp`), the stream's norms around zero,
    those of a sublayer's output near -0.5 so that the stream grows slowly; sinks N(0, 1); forget gates' biases spread
    over memories from a few tokens to hundreds, input gates' over a few units; router rows three times the usual size
    (so that choices are not close calls) with biases 0.5 N; rounded to `dtype`."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".", 1)[1] if name[0] == "l" and "." in name else name
        noise = torch.randn(shape, generator=gen)
        if leaf in ("norm1b", "norm2b"):
            t = 0.1 * noise - 0.5
        elif leaf in ("norm1", "norm2", "final.norm") or name == "final.norm":
            t = 0.2 * noise
        elif leaf.endswith("norm"):
            t = (1.0 + 0.2 * noise) * (sharp if leaf in ("mix.q.norm", "mix.dq.norm") else 1.0)
        elif leaf == "mix.sink":
            t = noise
        elif leaf == "mix.f.b":
            t = 3.0 + 1.5 * noise
        elif leaf == "mix.i.b":
            t = noise - 0.5
        elif leaf == "mlp.router.b":
            t = 0.5 * noise
        elif name in ("embed", "bigram", "pos"):
            t = noise
        else:
            t = noise * ((3.0 if leaf == "mlp.router" else 1.0) / shape[1] ** 0.5)
        out[name] = t.to(dtype)
    return out


def write_model_dir(folder: str, cfg: dict, weights: dict) -> str:
    from safetensors.torch import save_file

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(folder, "model.safetensors"))
    return folder


def random_tokens(cfg: dict, length: int, seed: int) -> list[int]:
    gen = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (length,), generator=gen).tolist()


# Largest |difference| over largest |expected| of a row of logits, against the plain implementation in float64. The
# float32 engine is the sharp comparison. In bfloat16 the engine rounds activations at some ten places a layer; those
# runs hold most positions to the bar and none beyond a loose one.
TOLERANCE = {"float32": 2e-4, "bfloat16": 6e-2}


def relative_error(got: torch.Tensor, want: torch.Tensor) -> float:
    return float((got.double() - want.double()).abs().max() / want.double().abs().max())


class TinyZemarax:
    """A configuration with random weights rounded to the engine's dtype (so that the plain implementation, which runs
    in float64, and the engine start from identical numbers), its model folder, and the plain implementation's logits
    on demand. `sharp` multiplies every score: with 3 or more a softmax rests on a few keys anywhere in reach, so that one
    key too many or too few moves the logits by far more than a rounding."""

    def __init__(self, key: str, dtype: str, seed: int = 1, cfg: dict | None = None, weights: dict | None = None,
                 page: int = 16, sharp: float = 1.0):
        if cfg is None:
            cfg, page = CONFIGS[key]
        self.cfg, self.page = cfg, page
        self.dtype = dtype
        torch_dtype = torch.float32 if dtype == "float32" else torch.bfloat16
        self.weights = weights if weights is not None else random_weights(cfg, seed, torch_dtype, sharp)
        self.weights = {k: v.to(torch_dtype) for k, v in self.weights.items()}
        self.plain_weights = {k: v.double() for k, v in self.weights.items()}
        self._dir = tempfile.TemporaryDirectory()
        self.folder = write_model_dir(self._dir.name, self.cfg, self.weights)
        self._plain: dict[tuple, torch.Tensor] = {}

    def plain_logits(self, tokens) -> torch.Tensor:
        key = tuple(tokens)
        if key not in self._plain:
            self._plain[key] = plain_zemarax.forward(self.cfg, self.plain_weights, list(tokens))
        return self._plain[key]

    def runner(self, n_pages: int, slots: int = 4, page: int | None = None):
        from pulsarlm_b200.cache.manager import CacheManager
        from pulsarlm_b200.engine.loading import load_model
        from pulsarlm_b200.engine.runner import ModelRunner

        model = load_model(self.folder, self.dtype, "cuda:0")
        cache = CacheManager(model.cache_needs(), page or self.page, n_pages, slots, model.ctx.dtype, "cuda:0")
        return ModelRunner(model, cache)

    def check(self, request_tokens: dict, got: dict, what: str) -> float:
        """Every returned row against the plain implementation's row at that position. float32: every position within
        the bar. bfloat16: every position within a loose bar and the median of a request's positions within half the
        bar; where the model routes tokens to experts, a few positions a request may lie beyond the loose bar (a
        rounding can tip a router's close call, which moves a row, and through the recurrent state those after it, by
        more than a rounding; the float32 run of the same schedule holds every position)."""
        worst = 0.0
        loose = self.dtype == "bfloat16"
        bar = 0.25 if loose else TOLERANCE[self.dtype]
        routes = any((entry.get("mlp") or {}).get("kind") == "moe" for entry in self.cfg["layers"])
        for r, rows in got.items():
            ref = self.plain_logits(request_tokens[r])
            errors = {position: relative_error(rows[position], ref[position]) for position in sorted(rows)}
            beyond = [(position, err) for position, err in errors.items() if err >= bar]
            allowed = max(1, len(rows) // 25) if loose and routes else 0
            assert len(beyond) <= allowed, (f"{what}: request {r!r} differs from the plain implementation at positions "
                                            f"{beyond[:5]} of {len(request_tokens[r])} (rel error; bar {bar:.0e})")
            middle = sorted(errors.values())[len(errors) // 2]
            if loose:
                assert middle < TOLERANCE["bfloat16"], f"{what}: request {r!r}: median error {middle:.3e}"
            worst = max(worst, *errors.values())
        return worst
