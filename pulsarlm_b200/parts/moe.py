"""A routed feed-forward: many small feed-forwards (gated, or plain with the square of relu or GELU)
of which each token uses a few, chosen by a router, beside an optional one that every token uses."""

from __future__ import annotations

import os

import torch

from ..kernels import ops
from .branches import run_branches
from .linear import activated_linear, gated_feed_forward, linear
from .registry import BuildContext, Part, register_part
from .spec import PartSpec, TensorNeed

# From this many tokens a bfloat16 step sorts its (token, expert) pairs by expert and runs the
# experts as grouped matrix products; below, every pair streams its expert's weights.
GROUPED_MIN_TOKENS = int(os.environ.get("PULSARLM_B200_MOE_GROUPED_MIN_TOKENS", "48"))


@register_part("feed_forward", "moe")
class RoutedExperts(Part):
    """Router (fp32): z = Wr h, s = softmax(z) over all experts, choice scores c = s +
    correction; experts form `groups` equal groups of neighbours, a group's score is its
    largest choice score and only experts of the `keep_groups` best groups can be chosen; the
    `top` largest choice scores are chosen and weigh in with s / (sum of the chosen s + 1e-20).
    Expert e: W_down,e (silu(W_gate,e h) * (W_up,e h)), no biases. The output is the weighted
    sum of the chosen experts' outputs plus, where `shared_size` is given, a shared expert of
    the same form that every token uses.

    Steps of few tokens (and the float32 engine) run the chosen experts pair by pair
    (csrc/moe.cu: every (token, expert) pair streams its expert's weights, sums in fp32,
    nothing depends on the rest of the batch). Longer bfloat16 steps sort the pairs by expert
    on the device and run each projection as one grouped matrix product over the sorted rows.
    No step asks the host which experts were chosen, so steps of single tokens can be
    captured.

    Variants, all parameters: `scores` = "sigmoid" makes s the sigmoid of every logit alone
    (default "softmax"); `group_top` = n makes a group's score the sum of its n largest choice
    scores (default 1); `renormalise` = False leaves the chosen scores as the weights (default
    True); `expert` = "relu2" makes every expert, and the shared one, W_down relu(W_up h)^2 without
    a gate (default "gated_silu"; such experts have no `expert_gate` / `shared_gate` tensors), "gelu" the same with the
    exact GELU. The tensor `logit_bias` [E], where given, joins the router's logits (choice and weights see it; with
    softmax scores and `renormalise` the weights are the softmax over the chosen experts' logits alone).

    `expert` = "clamped" gives experts the clamped unit in the place of silu(gate) * up (ops.gated_act) with
    `expert_limit`, and the shared expert `shared_limit`; `weigh_input` = True puts an expert's weight on its input
    instead of its output (on the gate and up products, which a linear map makes the same thing); the tensor
    `shared_gate_row` [1, H], where given, makes the shared expert join times sigmoid of its product with h (fp32,
    a row more in the router's kernel).

    params: hidden_size, expert_size, n_experts, top, groups (default 1), keep_groups
    (default groups), shared_size (optional), scores, group_top, renormalise, expert, expert_limit, shared_limit,
    weigh_input. tensors: router [E, H], correction [E] and logit_bias [E]
    (optional), experts: a name pattern with `{e}` for gate / up / down
    (`expert_gate`, `expert_up` [F, H], `expert_down` [H, F]), shared_gate, shared_up [Fs, H],
    shared_down [H, Fs]."""

    def __init__(self, spec: PartSpec, ctx: BuildContext):
        super().__init__(spec, ctx)
        p = spec.params
        self.hidden = int(self.param("hidden_size"))
        self.ff = int(self.param("expert_size"))
        self.n_experts = int(self.param("n_experts"))
        self.top = int(self.param("top"))
        self.groups = int(p.get("groups") or 1)
        self.keep = int(p.get("keep_groups") or self.groups)
        self.shared_size = int(p["shared_size"]) if p.get("shared_size") else 0
        self.sigmoid_scores = {"softmax": False, "sigmoid": True}[str(p.get("scores") or "softmax")]
        self.group_top = int(p.get("group_top") or 1)
        self.renormalise = bool(p.get("renormalise", True))
        expert = str(p.get("expert") or "gated_silu")
        self.gated = {"gated_silu": True, "relu2": False, "gelu": False, "clamped": True}[expert]
        self.plain_act = "gelu" if expert == "gelu" else "relu2"   # (experts without a gate)
        self.limit = float(self.param("expert_limit")) if expert == "clamped" else None
        self.shared_limit = float(self.param("shared_limit")) if expert == "clamped" and self.shared_size else None
        self.weigh_input = bool(p.get("weigh_input", False))
        if self.weigh_input and self.limit is None:
            raise ValueError("moe: only experts with the clamped unit take their weight on the input")
        self.shared_gate_row = bool(spec.tensors.get("shared_gate_row")) and self.shared_size > 0
        if self.n_experts % self.groups or not 0 < self.keep <= self.groups:
            raise ValueError(f"moe: {self.n_experts} experts in {self.groups} groups of which {self.keep} stay")
        if not 0 < self.top <= self.keep * (self.n_experts // self.groups):
            raise ValueError(f"moe: {self.top} experts cannot be chosen from {self.keep} groups of "
                             f"{self.n_experts // self.groups}")
        self.router = self.correction = self.logit_bias = None
        self.gate_up = self.down = None            # [E, 2F, H] ([E, F, H] without a gate), [E, H, F]
        self.gate_up_t = self.down_t = None        # the same with rows and columns swapped, for the grouped products
        self.shared_gate_up = self.shared_down = None

    @classmethod
    def tensor_needs(cls, spec: PartSpec) -> dict[str, TensorNeed]:
        p, t = spec.params, spec.tensors
        h, f, e = int(p["hidden_size"]), int(p["expert_size"]), int(p["n_experts"])
        gated = str(p.get("expert") or "gated_silu") in ("gated_silu", "clamped")
        needs = {t["router"]: TensorNeed((e, h))}
        if t.get("logit_bias"):
            needs[t["logit_bias"]] = TensorNeed((e,), role="offset")
        if t.get("correction"):
            needs[t["correction"]] = TensorNeed((e,), role="offset")
        for i in range(e):
            if gated:
                needs[t["expert_gate"].format(e=i)] = TensorNeed((f, h))
            needs[t["expert_up"].format(e=i)] = TensorNeed((f, h))
            needs[t["expert_down"].format(e=i)] = TensorNeed((h, f))
        if p.get("shared_size"):
            fs = int(p["shared_size"])
            if gated:
                needs[t["shared_gate"]] = TensorNeed((fs, h))
            needs[t["shared_up"]] = TensorNeed((fs, h))
            needs[t["shared_down"]] = TensorNeed((h, fs))
            if t.get("shared_gate_row"):
                needs[t["shared_gate_row"]] = TensorNeed((1, h))
        return needs

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        t = self.spec.tensors
        self.router = tensors[t["router"]].float().contiguous()
        if self.shared_gate_row:
            self.router = torch.cat([self.router, tensors[t["shared_gate_row"]].float()], dim=0).contiguous()
        self.correction = tensors[t["correction"]].float().contiguous() if t.get("correction") else None
        self.logit_bias = tensors[t["logit_bias"]].float().contiguous() if t.get("logit_bias") else None
        experts = range(self.n_experts)
        if self.gated:
            self.gate_up = torch.stack([torch.cat([tensors[t["expert_gate"].format(e=i)],
                                                   tensors[t["expert_up"].format(e=i)]], dim=0)
                                        for i in experts]).contiguous()
        else:
            self.gate_up = torch.stack([tensors[t["expert_up"].format(e=i)] for i in experts]).contiguous()
        self.down = torch.stack([tensors[t["expert_down"].format(e=i)] for i in experts]).contiguous()
        if self.shared_size:
            self.shared_gate_up = (torch.cat([tensors[t["shared_gate"]], tensors[t["shared_up"]]], dim=0).contiguous()
                                   if self.gated else tensors[t["shared_up"]].contiguous())
            self.shared_down = tensors[t["shared_down"]].contiguous()

    def _grouped(self, h: torch.Tensor) -> bool:
        return (h.dtype == torch.bfloat16 and h.shape[0] >= GROUPED_MIN_TOKENS and self.hidden % 8 == 0
                and self.ff % 8 == 0 and hasattr(torch.nn.functional, "grouped_mm"))

    def _route(self, h: torch.Tensor) -> tuple:
        """(ids, weights on the experts' inputs, weights on their outputs, weight of the shared expert); weights None: 1."""
        shared = torch.empty(h.shape[0], dtype=torch.float32, device=h.device) if self.shared_gate_row else None
        ids, weights = ops.moe_route(h, self.router, self.correction, self.top, self.groups, self.keep,
                                     self.sigmoid_scores, self.group_top, self.renormalise, shared, self.logit_bias)
        return (ids, weights, None, shared) if self.weigh_input else (ids, None, weights, shared)

    def _shared(self, h: torch.Tensor) -> torch.Tensor | None:
        """The shared expert's output."""
        if not self.shared_size:
            return None
        if self.gated:
            act = "silu" if self.shared_limit is None else "clamped"
            return gated_feed_forward(h, self.shared_gate_up, self.shared_down, act, self.shared_limit or 0.0)
        return activated_linear(linear(h, self.shared_gate_up), None, self.plain_act, self.shared_down)

    def _units(self, h: torch.Tensor) -> tuple:
        """Router and first half of the chosen experts, pair by pair: (activations [T * top, F], what `_route` says)."""
        routed = self._route(h)
        act = torch.empty((h.shape[0] * self.top, self.ff), dtype=h.dtype, device=h.device)
        if self.gated:
            ops.moe_gate_up(h, self.gate_up, routed[0], act, self.limit, routed[1])
        else:
            ops.moe_up(h, self.gate_up, routed[0], act, self.plain_act)
        return act, routed

    def forward(self, h: torch.Tensor, batch) -> torch.Tensor:
        out = torch.empty((h.shape[0], self.hidden), dtype=h.dtype, device=h.device)
        if not self._grouped(h):
            (act, (ids, _, weights, shared_weights)), shared = run_branches(
                batch, h.device, lambda: self._units(h), shared_expert=lambda: self._shared(h))
            ops.moe_down(act, self.down, ids, weights, shared, out, shared_weights)
            return out
        # Pairs in expert order; each projection one grouped product over the sorted rows (the library's: operands
        # [rows, K] and [E, K, N] with the experts' last rows as offsets).
        ids, in_weights, weights, shared_weights = self._route(h)
        shared = self._shared(h)
        ends, row_of_pair, pair_of_row = ops.moe_sort(ids, self.n_experts)
        x = ops.moe_gather(h, pair_of_row, self.top)
        gate_up = torch.nn.functional.grouped_mm(x, self.gate_up.transpose(1, 2), offs=ends)
        act = torch.empty((x.shape[0], self.ff), dtype=h.dtype, device=h.device)
        if self.limit is not None:
            ops.gated_act(gate_up, act, "clamped", self.limit, in_weights, pair_of_row)
        elif self.gated:
            ops.swiglu(gate_up, act)
        else:
            ops.bias_act(gate_up, None, act, self.plain_act)
        y = torch.nn.functional.grouped_mm(act, self.down.transpose(1, 2), offs=ends)
        ops.moe_combine(y, row_of_pair, weights, shared, out, shared_weights)
        return out
