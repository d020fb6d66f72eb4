"""Two mixers that read the same input, their outputs normed and averaged."""

from __future__ import annotations

import torch

from ..kernels import ops
from .basic import NormedSides
from .branches import run_branches
from .linear import linear
from .registry import BuildContext, Part, build_part, part_class, register_part
from .spec import PartSpec, TensorNeed


@register_part("mixer", "side_by_side")
class SideBySide(Part):
    """out = (rmsnorm(left(h)) * w_left + rmsnorm(right(h)) * w_right) / 2, both norms over the model width with one
    eps. The two mixers' projections of h are one product (their operands stacked at load; each mixer is handed its
    columns). A block that can carry it takes the outputs as a NormedSides (`pending`): the kernel that makes the next
    layer's input norms both, adds a side's last bias, and adds them into the stream in one pass.

    The left mixer is the one that keeps keys and values: the block's cache holders begin with this part, which stands
    for it; the right mixer and whatever either names besides follow as state holders.

    params: hidden_size, eps, left, right (PartSpecs of mixers that offer `projections` and `forward_columns`).
    tensors: left_norm, right_norm [H]."""

    def __init__(self, spec: PartSpec, ctx: BuildContext):
        super().__init__(spec, ctx)
        self.hidden = int(self.param("hidden_size"))
        self.eps = float(self.param("eps"))
        self.left = build_part("mixer", self.param("left"), ctx)
        self.right = build_part("mixer", self.param("right"), ctx)
        for side in (self.left, self.right):
            if not hasattr(side, "forward_columns"):
                raise ValueError(f"side_by_side: the mixer {side.spec.kind!r} cannot share a product with another")
        self.in_weight = self.left_weight = self.right_weight = None

    @classmethod
    def tensor_needs(cls, spec: PartSpec) -> dict[str, TensorNeed]:
        hidden = int(spec.params["hidden_size"])
        needs = {spec.tensors["left_norm"]: TensorNeed((hidden,), role="vector"),
                 spec.tensors["right_norm"]: TensorNeed((hidden,), role="vector")}
        for side in ("left", "right"):
            inner = spec.params[side]
            needs.update(part_class("mixer", inner.kind).tensor_needs(inner))
        return needs

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        t = self.spec.tensors
        self.left.load(tensors)
        self.right.load(tensors)
        self.left_weight = tensors[t["left_norm"]].float().contiguous()
        self.right_weight = tensors[t["right_norm"]].float().contiguous()
        self.in_weight = torch.cat([self.left.projections(), self.right.projections()], dim=0).contiguous()
        at = self.left.channels     # (the sides' operands are now rows of the stacked one)
        self.left.in_weight, self.right.in_weight = self.in_weight[:at], self.in_weight[at:]

    # ------------------------------------------------------------------ cache, planning
    def inner_parts(self) -> list:
        """The parts inside this one, for whoever asks all parts what they plan or note (they are loaded here)."""
        return [self.left, self.right]

    def cache_need(self):
        return self.left.cache_need()

    def cache_read_need(self):
        return self.left.cache_read_need()

    def bind_cache(self, binding) -> None:
        self.left.bind_cache(binding)

    def state_holders(self) -> list:
        return list(self.left.state_holders()) + [self.right] + list(self.right.state_holders())

    def captures_state_steps(self) -> bool:
        return True

    # ------------------------------------------------------------------ forward
    def pending(self, h: torch.Tensor, batch) -> NormedSides:
        """Both mixers' outputs as a residual contribution that is normed on its way in."""
        proj = linear(h, self.in_weight)
        at, stride = self.left.channels, self.in_weight.shape[0]
        left, right = run_branches(batch, h.device,
                                   lambda: self.left.forward_columns(proj[:, :at], stride, h, batch, True),
                                   right=lambda: self.right.forward_columns(proj[:, at:], stride, h, batch, True))
        return NormedSides(left, self.left.output_bias, self.left_weight, right, self.right.output_bias, self.right_weight,
                           0.5, self.eps)

    def forward(self, h: torch.Tensor, batch) -> torch.Tensor:
        sides = self.pending(h, batch)
        mixed = torch.zeros(h.shape, dtype=torch.float32, device=h.device)
        ops.side_norm(mixed, sides.sides(), sides.factor, sides.eps, None, None, 0.0, None)
        return mixed.to(h.dtype)
