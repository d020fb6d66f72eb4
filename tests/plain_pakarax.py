"""A plain, slow implementation of the Pakarax decoder in float64 torch on the CPU, one
function per mechanism, written from the architecture's equations. It shares no code
with the engine: whole sequences at once, no cache, no pages, no state slots.

Notation: x [T, W] the residual stream, h a layer's input (the normed stream), weights by
their checkpoint names ([out, in], applied as W h). `forward(..., rounding=torch.bfloat16)`
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


def filtered(u: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """y[t, c] = sum_j weight[c, j] * u[t - (taps - 1) + j, c], zeros before the sequence's start."""
    taps = weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    return sum(weight[:, j] * padded[j: j + u.shape[0]] for j in range(taps))


def query_temperature(positions: torch.Tensor, coef: float, every: int) -> torch.Tensor:
    """[T]: what a query at each position is multiplied by; it steps up once every `every` tokens."""
    return 1.0 + coef * torch.log(((positions + 1) // every).double() + 1.0)


def slopes(heads: int) -> list[float]:
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def sloped_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, sink: torch.Tensor | None) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv]; head h reads kv head h // (H / G); score (q . k) * scale
    minus the head's slope per token of distance; one more term exp(sink) in the denominator."""
    n, heads = q.shape[0], q.shape[1]
    per = heads // k.shape[1]
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    out = torch.zeros(n, heads, v.shape[-1], dtype=torch.float64)
    for h, slope in enumerate(slopes(heads)):
        s = (q[:, h] @ k[:, h // per].T) * scale - slope * (i - j)
        s = s.masked_fill(j > i, float("-inf"))
        if sink is not None:
            s = torch.cat([s, torch.full((n, 1), float(sink[h]), dtype=torch.float64)], dim=1)
        out[:, h] = torch.softmax(s, dim=-1)[:, :n] @ v[:, h // per]
    return out


def left_branch(h: torch.Tensor, w: dict, m: dict, positions: torch.Tensor, rnd) -> torch.Tensor:
    """Attention over filtered queries, keys and values."""
    n = h.shape[0]
    heads, kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (filtered(rnd(h @ w[name].T + w[name + ".b"]), w[name + ".conv"]) for name in ("q", "k", "v"))
    t = m.get("q_temp")
    if t:
        q = q * query_temperature(positions, float(t["coef"]), int(t["every"]))[:, None]
    q, k, v = rnd(q), rnd(k), rnd(v)
    a = sloped_attention(q.view(n, heads, dim), k.view(n, kv, dim), v.view(n, kv, vdim), float(m["scale"]), w["sink"])
    return rnd(rnd(a).reshape(n, heads * vdim) @ w["o"].T) + w["o.b"]


def linear_recurrence(u: torch.Tensor, w: dict, blocks: int, state: torch.Tensor | None = None) -> torch.Tensor:
    """u [T, width] -> the states [T, width]: r and i from block-diagonal maps of u, a = exp(-8 r softplus(lam)),
    S = a S + sqrt(1 - a^2) i u. `state`: the state before u[0] (None: zeros)."""
    n, width = u.shape
    size = width // blocks
    parts = u.view(n, blocks, size)
    r = torch.sigmoid(torch.einsum("tbc,boc->tbo", parts, w["ra"]) + w["ra.b"]).reshape(n, width)
    i = torch.sigmoid(torch.einsum("tbc,boc->tbo", parts, w["ri"]) + w["ri.b"]).reshape(n, width)
    a = torch.exp(-8.0 * r * torch.log1p(torch.exp(w["lam"])))
    s = torch.zeros(width, dtype=torch.float64) if state is None else state
    out = []
    for t in range(n):
        s = a[t] * s + torch.sqrt(1.0 - a[t] ** 2) * i[t] * u[t]
        out.append(s)
    return torch.stack(out)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def right_branch(h: torch.Tensor, w: dict, m: dict, rnd) -> torch.Tensor:
    """The recurrent branch: a filtered projection through the recurrence, times a GELU branch."""
    y = gelu_tanh(rnd(h @ w["y"].T + w["y.b"]))
    u = rnd(filtered(rnd(h @ w["x"].T + w["x.b"]), w["conv"]) + w["conv.b"])
    return rnd(rnd(linear_recurrence(u, w, m["blocks"]) * y) @ w["o"].T)


def side_by_side(left: torch.Tensor, right: torch.Tensor, w_left: torch.Tensor, w_right: torch.Tensor, eps: float) -> torch.Tensor:
    return 0.5 * (rms(left, eps) * w_left + rms(right, eps) * w_right)


def clamped_unit(gate: torch.Tensor, up: torch.Tensor, limit: float) -> torch.Tensor:
    """The gate cut off above at `limit`, the other factor on both sides; g sigmoid(1.702 g) (u + 1)."""
    g = gate.clamp(max=limit)
    return g * torch.sigmoid(1.702 * g) * (up.clamp(-limit, limit) + 1.0)


def clamped_ff(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, limit: float, rnd) -> torch.Tensor:
    return rnd(rnd(clamped_unit(rnd(h @ gate.T), rnd(h @ up.T), limit)) @ down.T)


def route(h: torch.Tensor, router: torch.Tensor, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """ids [T, top] and weights [T, top]: the largest sigmoid scores, which are the weights as they are."""
    s = torch.sigmoid(h @ router.T)
    ids = s.topk(top, dim=-1).indices
    return ids, s.gather(1, ids)


def routed_ff(h: torch.Tensor, w: dict, mlp: dict, rnd) -> torch.Tensor:
    """Every chosen expert sees its weight times the token; a shared expert joins times a gate per token."""
    ids, weights = route(h, w["router"], mlp["router"]["top"])
    limit = float(mlp["expert"]["limit"])
    out = torch.zeros(h.shape[0], w["e0.down"].shape[0], dtype=torch.float64)
    for t in range(h.shape[0]):
        for e, g in zip(ids[t].tolist(), weights[t].tolist()):
            unit = clamped_unit(g * (h[t] @ w[f"e{e}.gate"].T), g * (h[t] @ w[f"e{e}.up"].T), limit)
            out[t] += rnd(unit) @ w[f"e{e}.down"].T
    if mlp.get("shared"):
        shared = clamped_ff(h, w["shared.gate"], w["shared.up"], w["shared.down"], float(mlp["shared"]["limit"]), rnd)
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * shared
    return rnd(out)


def sub(weights: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def layer_runs(cfg: dict) -> list[tuple[int, bool]]:
    """(layer, whether a pass of the loop begins with it) in the order the layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    start, stop = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(start)]
    for _ in range(loop["times"]):
        runs += [(i, i == start) for i in range(start, stop)]
    return runs + [(i, False) for i in range(stop, n)]


def capped(logits: torch.Tensor, cap: float | None) -> torch.Tensor:
    return logits if not cap else cap * torch.tanh(logits / cap)


def forward(cfg: dict, weights: dict, tokens: list[int], rounding=None, streams: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence. weights: float64 tensors by checkpoint name.
    `streams`, if a list, receives the residual stream after every layer run."""
    def rnd(t: torch.Tensor) -> torch.Tensor:
        return t.to(rounding).to(torch.float64) if rounding is not None else t

    eps = float(cfg["norm"]["eps"])
    positions = torch.arange(len(tokens))
    x = entered = weights["embed"][torch.tensor(tokens)]
    for i, begins_pass in layer_runs(cfg):
        if begins_pass:
            x = rnd(torch.cat([x, entered], dim=1)) @ weights["loop.in"].T
        layer, p = cfg["layers"][i], f"l{i}."
        h = rnd(rms(x, eps) * weights[p + "norm1"])
        m = layer["mixer"]
        left = left_branch(h, sub(weights, p + "mix.left."), m["left"], positions, rnd)
        right = right_branch(h, sub(weights, p + "mix.right."), m["right"], rnd)
        add = side_by_side(left, right, weights[p + "mix.left.out"], weights[p + "mix.right.out"], eps)
        mlp = layer.get("mlp")
        if mlp:
            w = sub(weights, p + "mlp.")
            add = add + (routed_ff(h, w, mlp, rnd) if mlp["kind"] == "moe" else
                         clamped_ff(h, w["gate"], w["up"], w["down"], float(mlp["limit"]), rnd))
        x = x + add
        if streams is not None:
            streams.append(x.clone())
    h = rnd(rms(x, eps) * weights["final.norm"])
    return capped((h @ weights["head"].T) * float(cfg.get("logit_scale", 1.0)), cfg.get("logit_softcap"))
