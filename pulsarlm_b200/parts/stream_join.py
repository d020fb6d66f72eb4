"""The stream joined again with what entered the first layer, by a projection."""

from __future__ import annotations

import torch

from ..kernels import ops
from .basic import NormedSides, settle_pending
from .linear import linear
from .registry import BuildContext, Part, register_part
from .spec import PartSpec, TensorNeed


@register_part("join", "concat_linear")
class ConcatLinear(Part):
    """x <- W [x; x0], x the residual stream with whatever is pending added first and x0 the stream as it entered the
    first layer. One kernel adds what is pending and lays the two rows side by side in the engine's dtype; the
    product's fp32 accumulators become the new stream. params: hidden_size. tensors: weight [H, 2 H], the columns of x
    first."""

    def __init__(self, spec: PartSpec, ctx: BuildContext):
        super().__init__(spec, ctx)
        self.hidden = int(self.param("hidden_size"))
        self.weight: torch.Tensor | None = None

    @classmethod
    def tensor_needs(cls, spec: PartSpec) -> dict[str, TensorNeed]:
        hidden = int(spec.params["hidden_size"])
        return {spec.tensors["weight"]: TensorNeed((hidden, 2 * hidden))}

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        self.weight = tensors[self.spec.tensors["weight"]].contiguous()

    def forward(self, x: torch.Tensor, delta, entered: torch.Tensor) -> torch.Tensor:
        both = torch.empty((x.shape[0], 2 * self.hidden), dtype=self.ctx.dtype, device=x.device)
        if isinstance(delta, NormedSides):
            ops.side_norm(x, delta.sides(), delta.factor, delta.eps, delta.y3, None, 0.0, both, entered=entered)
        else:
            settle_pending(x, delta)
            ops.side_norm(x, None, 0.0, 0.0, None, None, 0.0, both, entered=entered)
        return linear(both, self.weight, out_dtype=torch.float32)
