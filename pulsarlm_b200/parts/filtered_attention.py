"""Grouped-query attention over queries, keys and values that each pass a short convolution over time, with a linear
bias by distance, an optional learned sink per head and an optional temperature on the queries."""

from __future__ import annotations

import math

import torch

from ..kernels import ops
from .attention import Attention
from .delta_rule import sequence_rows_plan
from .gated_delta import FilterState
from .linear import linear
from .registry import BuildContext, register_part
from .spec import KVCacheNeed, PartSpec, TensorNeed


def geometric_slopes(heads: int, octaves: float) -> list[float]:
    """2^(-octaves (h + 1) / heads) for head h: what a key is marked down per token of distance."""
    return [2.0 ** (-octaves * (h + 1) / heads) for h in range(heads)]


def stacked_rows(parts: list[torch.Tensor], multiple: int = 8) -> tuple[torch.Tensor, list[int]]:
    """The matrices of several projections of one input as one operand, each part starting on a row that is a
    multiple of `multiple` (rows of zeros in between, so that the product's columns of a part start on whole 16-byte
    pieces), and the parts' first rows."""
    out, starts, at = [], [], 0
    for part in parts:
        starts.append(at)
        out.append(part)
        at += part.shape[0]
        if at % multiple:
            out.append(torch.zeros((multiple - at % multiple, *part.shape[1:]), dtype=part.dtype, device=part.device))
            at += multiple - at % multiple
    return torch.cat(out, dim=0).contiguous(), starts


@register_part("mixer", "filtered_attention")
class FilteredAttention(Attention):
    """With h the mixer's input:

        u = W h + b                                           for each of q, k and v (biases optional)
        y[t] = sum_j c[:, j] * u[t - (taps - 1) + j]           per channel, zeros before the sequence's start
        q = y_q * (1 + coef * ln(floor((p + 1) / every) + 1))  at position p (`temperature`, optional)
        a_h = softmax attention of q_h over k_g, v_g (g = h // (heads / kv_heads)), scores (q . k) * scale minus
              slope_h per token of distance (`slope_octaves`, see `geometric_slopes`), one more term exp(sink_h) in
              the denominator (the `sink` tensor, optional)
        out = Wo a (+ bo)

    Key and value sizes may differ: q, k and v are laid out as rows of a common size (the larger, rounded up to a
    multiple of 16, zeros past a row's own columns), so that the paged attention kernels, which know one row size, run
    them as they are; Wo gets zero columns to match. The cache holds filtered keys and values; the last taps - 1
    projected rows of a request (before the bias) are a state slot of its own (`state_holders`). One kernel
    (csrc/conv_qkv.cu) lies between the projection and the attention kernels and moves the slot on in steps of single
    tokens.

    `projections()` and `forward_columns` let a caller make this mixer's projections together with others of the same
    input; `output_bias` is left to a caller that takes it (`bias_taken`).

    params: hidden_size, n_heads, n_kv_heads, head_dim (keys), value_dim, taps, scale, window, slope_octaves (None: no
    bias), temperature ((coef, every) or None), split_weights. tensors: q [nh*hd, H], k [nkv*hd, H], v [nkv*vd, H], o
    [H, nh*vd], q_conv, k_conv, v_conv [channels, taps]; optional q_bias, k_bias, v_bias, o_bias, sink [nh]."""

    def __init__(self, spec: PartSpec, ctx: BuildContext):
        p = spec.params
        self.key_dim = int(p["head_dim"])
        self.value_dim = int(p.get("value_dim") or self.key_dim)
        self.row = -(-max(self.key_dim, self.value_dim) // 16) * 16
        scale = float(p["scale"]) if p.get("scale") is not None else 1.0 / math.sqrt(self.key_dim)
        inner = PartSpec(spec.kind, {**p, "head_dim": self.row, "scale": scale, "position": PartSpec("none")}, spec.tensors)
        super().__init__(inner, ctx)
        self.spec = spec
        if p.get("cache_from") is not None or p.get("softcap") or p.get("sink_logit") is not None:
            raise ValueError("filtered_attention: cache_from, softcap and constant sinks are not supported")
        self.taps = int(self.param("taps"))
        if not 1 <= self.taps <= 16:
            raise ValueError(f"filtered_attention: taps must be 1 to 16, got {self.taps}")
        self.temp_coef, self.temp_every = 0.0, 1
        if p.get("temperature") is not None:
            self.temp_coef, self.temp_every = float(p["temperature"][0]), int(p["temperature"][1])
            if self.temp_every <= 0:
                raise ValueError(f"filtered_attention: the temperature's step must be positive, got {self.temp_every}")
        if p.get("slope_octaves") is not None:
            self.distance_slopes = torch.tensor(geometric_slopes(self.n_heads, float(p["slope_octaves"])),
                                                dtype=torch.float32, device=ctx.device)
        self.sizes = (self.n_heads * self.key_dim, self.n_kv * self.key_dim, self.n_kv * self.value_dim)
        starts, at = [], 0
        for size in self.sizes:
            starts.append(at)
            at += -(-size // 8) * 8
        self.starts, self.channels = starts, at   # columns of q, k, v (each on a whole 16-byte piece), and all of them
        self.filter_state = FilterState(self.taps, self.channels)
        self.bias = self.conv = self.output_bias = None
        self.in_weight: torch.Tensor | None = None

    @classmethod
    def tensor_needs(cls, spec: PartSpec) -> dict[str, TensorNeed]:
        p, t = spec.params, spec.tensors
        h, nh, nkv, hd = (int(p[k]) for k in ("hidden_size", "n_heads", "n_kv_heads", "head_dim"))
        vd, taps = int(p.get("value_dim") or hd), int(p["taps"])
        needs = {t["o"]: TensorNeed((h, nh * vd))}
        for name, rows in (("q", nh * hd), ("k", nkv * hd), ("v", nkv * vd)):
            needs[t[name]] = TensorNeed((rows, h))
            needs[t[name + "_conv"]] = TensorNeed((rows, taps))
            if t.get(name + "_bias"):
                needs[t[name + "_bias"]] = TensorNeed((rows,), role="offset")
        if t.get("o_bias"):
            needs[t["o_bias"]] = TensorNeed((h,), role="offset")
        if t.get("sink"):
            needs[t["sink"]] = TensorNeed((nh,), role="offset")
        return needs

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        t = self.spec.tensors
        names = ("q", "k", "v")
        self.in_weight, starts = stacked_rows([tensors[t[n]] for n in names])
        assert starts == self.starts and self.in_weight.shape[0] == self.channels
        self.conv = stacked_rows([tensors[t[n + "_conv"]].float() for n in names])[0].t().contiguous()   # [taps, channels]
        if any(t.get(n + "_bias") for n in names):
            self.bias = stacked_rows([tensors[t[n + "_bias"]].float() if t.get(n + "_bias") else
                                      torch.zeros(size, device=self.ctx.device)
                                      for n, size in zip(names, self.sizes)])[0]
        o = tensors[t["o"]]
        if self.row != self.value_dim:
            padded = torch.zeros((self.hidden, self.n_heads, self.row), dtype=o.dtype, device=o.device)
            padded[:, :, :self.value_dim] = o.view(self.hidden, self.n_heads, self.value_dim)
            o = padded.view(self.hidden, self.n_heads * self.row)
        self.o = o.contiguous()
        self.output_bias = tensors[t["o_bias"]].float().contiguous() if t.get("o_bias") else None
        self.sinks = tensors[t["sink"]].float().contiguous() if t.get("sink") else None

    def cache_need(self) -> KVCacheNeed:
        return KVCacheNeed(self.n_kv, self.row, self.window, self.n_heads)

    def cache_read_need(self) -> KVCacheNeed:
        return self.cache_need()

    def state_holders(self) -> list:
        """What else keeps something per request for this mixer: the convolutions' inputs."""
        return [self.filter_state]

    def captures_state_steps(self) -> bool:
        return True

    def plan_key(self):
        key = super().plan_key()
        return ("filtered", *key) if key is not None else None

    def plan_step(self, step) -> dict:
        """What attention plans, and the rows of every entry (for the convolutions' slots)."""
        return {**super().plan_step(step), **sequence_rows_plan(step)}

    def _folds_rope(self, tokens, batch, inv_freq, rotary) -> bool:
        return False  # (nothing is rotated; the convolution is a kernel of its own)

    def native_choice(self, tokens, batch, row_stride):
        return None

    def projections(self) -> torch.Tensor:
        """The operand of this mixer's projections of its input, [rows, H] (see `stacked_rows`)."""
        return self.in_weight

    def forward_columns(self, proj: torch.Tensor, row_stride: int, h: torch.Tensor, batch, bias_taken: bool) -> torch.Tensor:
        """The mixer from its projections: proj [T, channels], columns of a matrix whose rows are `row_stride` apart."""
        tokens = proj.shape[0]
        cache = self.cache
        table = batch.tables[cache.group]
        q = torch.empty((tokens, self.n_heads, self.row), dtype=proj.dtype, device=proj.device)
        states = self.filter_state.states(proj)
        single = int(batch.n_decode) == tokens                 # every entry brings one token
        ops.conv_qkv_write(proj, row_stride, self.bias, self.conv, states, batch.slots, single, self.temp_coef,
                           self.temp_every, batch.pos, batch.entry, table, q, cache.k_pool, cache.v_pool, cache.page_size,
                           self.n_kv, self.key_dim, self.value_dim, self.starts[1], self.starts[2], batch.status)
        if self.taps > 1 and not single:
            plan = batch.plans[self.plan_key()]
            ops.filter_state(proj, row_stride, plan["first"], plan["count"], batch.slots, states)
        out = torch.empty((tokens, self.n_heads, self.row), dtype=proj.dtype, device=proj.device)
        self.attend(q, out, table, batch)
        y = linear(out.view(tokens, self.n_heads * self.row), self.o)
        if self.output_bias is not None and not bias_taken:
            ops.bias_act(y, self.output_bias.to(y.dtype), y, "none")
        return y

    def forward(self, h: torch.Tensor, batch) -> torch.Tensor:
        proj = linear(h, self.in_weight)
        return self.forward_columns(proj, proj.stride(0), h, batch, False)
