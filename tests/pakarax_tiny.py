"""Small Pakarax configurations and random weights for the tests.

The configurations differ from each other in every size and constant: layer order, widths, head counts (query heads per
kv head 1, 2, 3 and 4), key sizes above and below the value size, taps of the two branches (also 1, also unlike each
other), recurrence widths above and below the model's and gate blocks of odd and even sizes, layers with a temperature
on the queries and without, dense and routed feed-forwards (with and without a shared expert, one chosen expert and
several, limits that bite), a layer without feed-forward, loops that begin with the first layer or later, no loop,
logit scales and caps (also none). Weights are drawn with torch and written with the `safetensors` package, so the
engine's reader and its names are checked against an independent file.
"""

from __future__ import annotations

import json
import os
import tempfile

import torch

import plain_pakarax


def dense(ff, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def routed(ff, experts, top, limit=1.0, shared=None):
    """shared: (ff, limit) or None."""
    mlp = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared[0], "limit": shared[1]}
    return mlp


def layer(heads, kv_heads, dim, vdim, conv, width, blocks, right_conv, mlp, temp=(0.4, 16), scale=None):
    """temp: (coef, every) or None."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
            "scale": scale if scale is not None else 1.5 * dim ** -0.5}
    if temp:
        left["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "parallel", "mixer": {"left": left, "right": {"width": width, "blocks": blocks, "conv": right_conv}},
            "mlp": mlp}


def config(vocab, width, eps, logit_scale, softcap, loop, layers):
    """softcap: a number or None; loop: (start, stop, times) or None."""
    cfg = {"architecture": "Pakarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
           "layers": layers}
    if softcap is not None:
        cfg["logit_softcap"] = softcap
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


CONFIG_A = config(211, 72, 1e-5, 1.5, 8.0, (0, 2, 3), [
    layer(4, 2, 16, 24, 4, 48, 3, 2, dense(96)),
    layer(6, 2, 24, 8, 3, 80, 1, 4, routed(24, 8, 2, 0.8, (40, 0.7)), temp=(0.25, 7)),
    layer(2, 2, 16, 16, 1, 24, 2, 3, None, temp=None),
])
CONFIG_B = config(97, 40, 1e-3, 1.0, None, None, [
    layer(3, 1, 8, 8, 3, 20, 4, 5, routed(16, 5, 3), temp=None, scale=0.6),
    layer(4, 4, 12, 20, 2, 60, 5, 1, None, temp=(0.9, 1)),
    layer(5, 5, 10, 6, 6, 33, 3, 4, dense(50, 0.6)),
])
CONFIG_C = config(128, 64, 1e-6, 0.7, 5.0, (1, 3, 2), [
    layer(4, 2, 64, 64, 3, 64, 2, 4, dense(80)),
    layer(3, 3, 64, 32, 2, 128, 4, 3, routed(32, 6, 1, 1.2, (48, 0.9))),
    layer(4, 1, 80, 128, 4, 96, 3, 2, routed(48, 4, 2, 0.7), temp=(0.5, 40)),
    layer(8, 2, 32, 48, 3, 32, 1, 3, dense(72, 2.5), temp=None),
])
CONFIGS = {"A": (CONFIG_A, 16), "B": (CONFIG_B, 32), "C": (CONFIG_C, 16)}


def tensor_shapes(cfg: dict) -> dict[str, tuple[int, ...]]:
    w = cfg["width"]
    shapes = {"embed": (cfg["vocab"], w), "head": (cfg["vocab"], w), "final.norm": (w,)}
    if cfg.get("loop"):
        shapes["loop.in"] = (w, 2 * w)
    for i, entry in enumerate(cfg["layers"]):
        p, a, r = f"l{i}.", entry["mixer"]["left"], entry["mixer"]["right"]
        shapes[p + "norm1"] = (w,)
        rows = {"q": a["heads"] * a["dim"], "k": a["kv_heads"] * a["dim"], "v": a["kv_heads"] * a["vdim"]}
        for n, size in rows.items():
            shapes[p + f"mix.left.{n}"], shapes[p + f"mix.left.{n}.b"] = (size, w), (size,)
            shapes[p + f"mix.left.{n}.conv"] = (size, a["conv"])
        shapes[p + "mix.left.sink"] = (a["heads"],)
        shapes[p + "mix.left.o"], shapes[p + "mix.left.o.b"] = (w, a["heads"] * a["vdim"]), (w,)
        width, block = r["width"], r["width"] // r["blocks"]
        for n in ("y", "x"):
            shapes[p + f"mix.right.{n}"], shapes[p + f"mix.right.{n}.b"] = (width, w), (width,)
        shapes[p + "mix.right.conv"], shapes[p + "mix.right.conv.b"] = (width, r["conv"]), (width,)
        for n in ("ra", "ri"):
            shapes[p + f"mix.right.{n}"] = (r["blocks"], block, block)
            shapes[p + f"mix.right.{n}.b"] = (r["blocks"], block)
        shapes[p + "mix.right.lam"], shapes[p + "mix.right.o"] = (width,), (w, width)
        shapes[p + "mix.left.out"], shapes[p + "mix.right.out"] = (w,), (w,)
        mlp = entry["mlp"]
        if mlp is None:
            continue
        units = {"": mlp["ff"]} if mlp["kind"] == "dense" else {f"e{e}.": mlp["expert"]["ff"]
                                                                  for e in range(mlp["router"]["experts"])}
        if mlp["kind"] == "moe":
            shapes[p + "mlp.router"] = (mlp["router"]["experts"], w)
            if mlp.get("shared"):
                units["shared."] = mlp["shared"]["ff"]
                shapes[p + "mlp.shared.sg"] = (1, w)
        for n, ff in units.items():
            shapes[p + f"mlp.{n}gate"], shapes[p + f"mlp.{n}up"], shapes[p + f"mlp.{n}down"] = (ff, w), (ff, w), (w, ff)
    return shapes


def random_weights(cfg: dict, seed: int, dtype: torch.dtype = torch.float32) -> dict:
    """Matrices N(0, 1/sqrt(in)), norm weights 1 + 0.2 N (the stream's norms 0.5 + 0.1 N), biases 0.3 N, taps N(0,
    1/sqrt(taps)), sinks N(0, 1), decays from a few tokens' reach to a thousand's (lambda in (-9, 0)), gates twice the
    usual size, router rows three times (so that choices are not close calls); rounded to `dtype`."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".", 1)[1] if name[0] == "l" and "." in name and name != "loop.in" else name
        draw = torch.randn(shape, generator=gen)
        if leaf == "norm1":
            t = 0.5 + 0.1 * draw
        elif leaf in ("final.norm", "mix.left.out", "mix.right.out"):
            t = 1.0 + 0.2 * draw
        elif leaf.endswith(".b"):
            t = 0.3 * draw
        elif leaf.endswith("conv"):
            t = draw / shape[1] ** 0.5
        elif leaf == "mix.right.lam":
            t = -9.0 * torch.rand(shape, generator=gen)
        elif leaf == "mix.left.sink" or name == "embed":
            t = draw
        elif leaf in ("mix.right.ra", "mix.right.ri"):
            t = 2.0 * draw / shape[2] ** 0.5
        else:
            t = draw * ((3.0 if leaf == "mlp.router" else 1.0) / shape[-1] ** 0.5)
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


def sharpened(cfg: dict, sharp: float) -> dict:
    """The configuration with every layer's score scale times `sharp`: with 3 or more a softmax rests on a few keys
    anywhere in reach, so that one key too many or too few moves the logits by far more than a rounding."""
    cfg = json.loads(json.dumps(cfg))
    for entry in cfg["layers"]:
        entry["mixer"]["left"]["scale"] *= sharp
    return cfg


class TinyPakarax:
    """A configuration with random weights rounded to the engine's dtype (so that the plain implementation, which runs
    in float64, and the engine start from identical numbers), its model folder, and the plain implementation's logits
    on demand."""

    def __init__(self, key: str, dtype: str, seed: int = 1, cfg: dict | None = None, weights: dict | None = None,
                 page: int = 16, sharp: float = 1.0):
        if cfg is None:
            cfg, page = CONFIGS[key]
        self.cfg, self.page = sharpened(cfg, sharp), page
        self.dtype = dtype
        torch_dtype = torch.float32 if dtype == "float32" else torch.bfloat16
        self.weights = weights if weights is not None else random_weights(self.cfg, seed, torch_dtype)
        self.weights = {k: v.to(torch_dtype) for k, v in self.weights.items()}
        self.plain_weights = {k: v.double() for k, v in self.weights.items()}
        self._dir = tempfile.TemporaryDirectory()
        self.folder = write_model_dir(self._dir.name, self.cfg, self.weights)
        self._plain: dict[tuple, torch.Tensor] = {}

    def plain_logits(self, tokens) -> torch.Tensor:
        key = tuple(tokens)
        if key not in self._plain:
            self._plain[key] = plain_pakarax.forward(self.cfg, self.plain_weights, list(tokens))
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
