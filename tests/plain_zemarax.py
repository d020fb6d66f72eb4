"""A plain, slow implementation of the Zemarax decoder in float64 torch on the CPU, one
function per mechanism, written from the architecture's equations. It shares no code
with the engine: whole sequences at once, no cache, no pages, no state slots.

Notation: x [T, W] the residual stream, h a sublayer's input (the normed stream), weights
by their checkpoint names ([out, in], applied as W h). `forward(..., rounding=torch.bfloat16)`
rounds where a bfloat16 engine stores a tensor (projections, cached rows, sublayer outputs),
so that the comparison with such an engine sees its arithmetic and not its storage.
"""

from __future__ import annotations

import math

import torch


def relative_error_of(got: torch.Tensor, want: torch.Tensor) -> float:
    """Largest |difference| over largest |wanted|."""
    return float((got.double() - want.double()).abs().max() / want.double().abs().max().clamp(min=1e-30))


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """The stream's norm: its weight is stored around zero."""
    return rms(x, eps) * (1.0 + weight)


def embedding(tokens: list[int], table: torch.Tensor, pairs: torch.Tensor | None, places: torch.Tensor | None, cfg: dict,
              before: int | None = None, start: int = 0) -> torch.Tensor:
    """table[token] * scale, plus a row of `pairs` chosen by a hash of (token before, token) (a sequence's first
    token takes the last row), plus the learned vector of the token's position; the scale touches the first
    term only. `before`: the token ahead of tokens[0] (None: a sequence's start), `start`: its position."""
    e = cfg.get("embedding") or {}
    x = table[torch.tensor(tokens)] * float(e.get("scale", 1.0))
    if pairs is not None:
        b = e["bigram"]
        rows = []
        for t, tok in enumerate(tokens):
            prev = tokens[t - 1] if t > 0 else before
            rows.append(b["buckets"] if prev is None else (prev * b["mul_prev"] + tok * b["mul_cur"]) % b["buckets"])
        x = x + pairs[torch.tensor(rows)]
    if places is not None:
        x = x + places[start: start + len(tokens)]
    return x


def in_reach(n: int, window: int | None, keep_first: int) -> torch.Tensor:
    """[n, n] bool: query i sees key j <= i if it is less than `window` tokens back or among the first `keep_first`."""
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    seen = j <= i
    if window is not None:
        seen = seen & ((i - j < window) | (j < keep_first))
    return seen


def sink_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, seen: torch.Tensor,
                   sink: torch.Tensor | None) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv]; head h reads kv head h // (H / G); scores (q . k) * scale where
    `seen`, one more term exp(sink_h) in the denominator."""
    n, heads = q.shape[0], q.shape[1]
    per = heads // k.shape[1]
    out = torch.zeros(n, heads, v.shape[-1], dtype=torch.float64)
    for h in range(heads):
        s = ((q[:, h] @ k[:, h // per].T) * scale).masked_fill(~seen, float("-inf"))
        if sink is not None:
            s = torch.cat([s, torch.full((n, 1), float(sink[h]), dtype=torch.float64)], dim=1)
        out[:, h] = torch.softmax(s, dim=-1)[:, :n] @ v[:, h // per]
    return out


def windowed_attention(h: torch.Tensor, w: dict, m: dict, eps: float, rnd) -> torch.Tensor:
    n, heads, kv, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = rnd(h @ w["q"].T).view(n, heads, dim), rnd(h @ w["k"].T).view(n, kv, dim), rnd(h @ w["v"].T).view(n, kv, vdim)
    q, k = rnd(rms(q, eps) * w["q.norm"]), rnd(rms(k, eps) * w["k.norm"])
    mask = m.get("mask") or {}
    a = sink_attention(q, k, v, float(m["scale"]), in_reach(n, mask.get("size"), mask.get("keep_first", 0)), w.get("sink"))
    return rnd(rnd(a).reshape(n, heads * vdim) @ w["o"].T)


def latent_of(h: torch.Tensor, w: dict, eps: float, rnd) -> torch.Tensor:
    """What a latent layer caches: [T, rank]."""
    return rnd(rms(rnd(h @ w["dkv"].T), eps) * w["dkv.norm"])


def latent_attention(h: torch.Tensor, w: dict, m: dict, eps: float, latent: torch.Tensor, rnd) -> torch.Tensor:
    n, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    cq = rnd(rms(rnd(h @ w["dq"].T), eps) * w["dq.norm"])
    q = rnd(cq @ w["uq"].T).view(n, heads, dim)
    k, v = (latent @ w["uk"].T).view(n, heads, dim), (latent @ w["uv"].T).view(n, heads, vdim)
    a = sink_attention(q, k, v, float(m["scale"]), in_reach(n, None, 0), w.get("sink"))
    return rnd(rnd(a).reshape(n, heads * vdim) @ w["o"].T)


def log_gates(i_pre: torch.Tensor, f_pre: torch.Tensor, cap: float) -> tuple[torch.Tensor, torch.Tensor]:
    """Log input gate and log forget gate, both from soft-capped logits (biases already added)."""
    i = cap * torch.tanh(i_pre / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh(f_pre / cap))
    return i, f


def matrix_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, i: torch.Tensor, f: torch.Tensor,
                  state: tuple | None = None) -> tuple[torch.Tensor, tuple]:
    """q (scaled), k [T, H, D], v [T, H, Dv], log gates [T, H] -> (o [T, H, Dv], state). State: S [H, D, Dv], n [H, D],
    m [H], all zero at a sequence's start."""
    steps, heads, dim = q.shape
    if state is None:
        state = (torch.zeros(heads, dim, v.shape[-1], dtype=q.dtype), torch.zeros(heads, dim, dtype=q.dtype),
                 torch.zeros(heads, dtype=q.dtype))
    s, n, m = (x.clone() for x in state)
    out = torch.empty_like(v)
    for t in range(steps):
        top = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - top), torch.exp(i[t] - top)
        s = keep[:, None, None] * s + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = top
        numerator = torch.einsum("hd,hde->he", q[t], s)
        denominator = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = numerator / denominator[:, None]
    return out, (s, n, m)


def matrix_memory_mixer(h: torch.Tensor, w: dict, m: dict, eps: float, rnd) -> torch.Tensor:
    n, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = rnd(h @ w["q"].T).view(n, heads, dim) * dim ** -0.5, rnd(h @ w["k"].T).view(n, heads, dim)
    v = rnd(h @ w["v"].T).view(n, heads, vdim)
    i, f = log_gates(h @ w["i"].T + w["i.b"], h @ w["f"].T + w["f.b"], float(m["gate_cap"]))
    o, _ = matrix_memory(q, k, v, i, f)
    o = rms(o, eps).reshape(n, heads * vdim) * w["norm"] * torch.sigmoid(rnd(h @ w["g"].T))
    return rnd(rnd(o) @ w["o"].T)


def gated_ff(h: torch.Tensor, w: dict, rnd) -> torch.Tensor:
    g = rnd(h @ w["gate"].T)
    return rnd(rnd(g * torch.sigmoid(g) * rnd(h @ w["up"].T)) @ w["down"].T)


def gelu(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def gelu_ff(h: torch.Tensor, up: torch.Tensor, down: torch.Tensor, rnd) -> torch.Tensor:
    return rnd(rnd(gelu(rnd(h @ up.T))) @ down.T)


def route(h: torch.Tensor, router: torch.Tensor, bias: torch.Tensor, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """ids [T, top] and weights [T, top]: the largest biased logits, and the softmax over those alone."""
    z, ids = (h @ router.T + bias).topk(top, dim=-1)
    return ids, torch.softmax(z, dim=-1)


def routed_ff(h: torch.Tensor, w: dict, mlp: dict, rnd) -> torch.Tensor:
    ids, weights = route(h, w["router"], w["router.b"], mlp["router"]["top"])
    out = torch.zeros(h.shape[0], w["e0.down"].shape[0], dtype=torch.float64)
    for e in range(mlp["router"]["experts"]):
        share = (weights * (ids == e)).sum(-1)
        rows = torch.nonzero(share > 0).flatten()
        if rows.numel():
            out[rows] += share[rows, None] * gelu_ff(h[rows], w[f"e{e}.up"], w[f"e{e}.down"], rnd)
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * gelu_ff(h, w["shared.up"], w["shared.down"], rnd)
    return rnd(out)


def sub(weights: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg: dict, weights: dict, tokens: list[int], rounding=None, streams: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence. weights: float64 tensors by checkpoint name.
    `streams`, if a list, receives the residual stream after every layer."""
    def rnd(t: torch.Tensor) -> torch.Tensor:
        return t.to(rounding).to(torch.float64) if rounding is not None else t

    eps = float(cfg["norm"]["eps"])
    x = embedding(tokens, weights["embed"], weights.get("bigram"), weights.get("pos"), cfg)
    latents: dict[int, torch.Tensor] = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rnd(offset_norm(x, weights[p + "norm1"], eps))
        w = sub(weights, p + "mix.")
        if layer["type"] == "attention":
            y = windowed_attention(h, w, m, eps, rnd)
        elif layer["type"] == "mlstm":
            y = matrix_memory_mixer(h, w, m, eps, rnd)
        else:
            if m.get("kv_from") is None:
                latents[i] = latent_of(h, w, eps, rnd)
            y = latent_attention(h, w, m, eps, latents[i if m.get("kv_from") is None else m["kv_from"]], rnd)
        x = x + offset_norm(y, weights[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp:
            h = rnd(offset_norm(x, weights[p + "norm2"], eps))
            w = sub(weights, p + "mlp.")
            y = routed_ff(h, w, mlp, rnd) if mlp["kind"] == "moe" else gated_ff(h, w, rnd)
            x = x + offset_norm(y, weights[p + "norm2b"], eps)
        if streams is not None:
            streams.append(x.clone())
    h = rnd(offset_norm(x, weights["final.norm"], eps))
    return (h @ weights["head"].T) * float(cfg.get("logit_scale", 1.0))
