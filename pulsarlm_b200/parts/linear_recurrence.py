"""A gated linear recurrence per channel (an RG-LRU: De et al., "Griffin: Mixing Gated Linear Recurrences with Local
Attention for Efficient Language Models") behind a short convolution, beside a GELU branch."""

from __future__ import annotations

import torch

from ..kernels import ops
from .delta_rule import SEQUENCE_ROWS_KEY, sequence_rows_plan
from .filtered_attention import stacked_rows
from .linear import linear
from .registry import BuildContext, Part, register_part
from .spec import PartSpec, StateNeed, TensorNeed


class RingState:
    """The last inputs of a convolution over time, per request: [taps, channels] in the engine's dtype (what the
    projection wrote, so a cut changes no bit), the input at position p in row p mod taps. One row more than the
    taps - 1 a token reads, so that the row a token writes is none of those any block of its kernel reads. A cache
    holder beside the mixer that owns it."""

    def __init__(self, taps: int, channels: int):
        self.taps, self.channels = taps, channels
        self.binding = None

    def cache_need(self) -> StateNeed:
        return StateNeed((self.taps, self.channels), dtype="engine")

    def bind_cache(self, binding) -> None:
        self.binding = binding

    def captures_state_steps(self) -> bool:
        return True


@register_part("mixer", "linear_recurrence")
class LinearRecurrence(Part):
    """With h the mixer's input and `width` channels in `blocks` equal blocks:

        y = gelu(Wy h + by)                                      (the tanh form)
        u = conv(Wx h + bx) + bc                                  causal, per channel, zeros before the start
        r, i = sigmoid(Ra_b u_b + ba_b), sigmoid(Ri_b u_b + bi_b) block by block
        log a = decay * r,  decay = -8 softplus(lambda)
        S <- a S + sqrt(1 - a^2) i u                              from S = 0, the first token too
        out = Wo (S * y)

    S is fp32 per request (this part's own state); the convolution's inputs are a RingState. Gates, decays and the
    recurrence are fp32. Steps of single tokens in bfloat16 run everything between the projections in one kernel;
    other steps run the convolution, the gates' block-diagonal products (one batched library product with fp32
    results; `gemm_f32` block by block in the float32 engine) and the scan (csrc/linear_recurrence.cu), whose sums are
    made in token order.

    params: hidden_size, width, blocks, taps, decay_scale (default 8). tensors: y, x [width, H], y_bias, x_bias
    [width], conv [width, taps], conv_bias [width], ra, ri [blocks, width / blocks, width / blocks], ra_bias, ri_bias
    [blocks, width / blocks], lam [width], o [H, width]."""

    output_bias = None

    def __init__(self, spec: PartSpec, ctx: BuildContext):
        super().__init__(spec, ctx)
        self.hidden = int(self.param("hidden_size"))
        self.width = int(self.param("width"))
        self.blocks = int(self.param("blocks"))
        self.taps = int(self.param("taps"))
        self.decay_scale = float(spec.params.get("decay_scale") or 8.0)
        if self.blocks < 1 or self.width % self.blocks:
            raise ValueError(f"linear_recurrence: {self.width} channels do not split into {self.blocks} blocks")
        if self.taps < 1:
            raise ValueError(f"linear_recurrence: taps must be at least 1, got {self.taps}")
        self.block = self.width // self.blocks
        self.column = -(-self.width // 8) * 8   # columns a branch takes of the projections' output
        self.channels = 2 * self.column
        self.in_weight = self.o = self.gates = self.conv = self.decay = None
        self.x_bias = self.y_bias = self.conv_bias = self.ra_bias = self.ri_bias = None
        self.states = None
        self.ring = RingState(self.taps, self.width)

    @classmethod
    def tensor_needs(cls, spec: PartSpec) -> dict[str, TensorNeed]:
        p, t = spec.params, spec.tensors
        h, width, blocks, taps = (int(p[k]) for k in ("hidden_size", "width", "blocks", "taps"))
        block = width // max(blocks, 1)
        needs = {t["y"]: TensorNeed((width, h)), t["x"]: TensorNeed((width, h)), t["conv"]: TensorNeed((width, taps)),
                 t["ra"]: TensorNeed((blocks, block, block)), t["ri"]: TensorNeed((blocks, block, block)),
                 t["o"]: TensorNeed((h, width))}
        for name in ("y_bias", "x_bias", "conv_bias", "lam"):
            needs[t[name]] = TensorNeed((width,), role="offset")
        for name in ("ra_bias", "ri_bias"):
            needs[t[name]] = TensorNeed((blocks, block), role="offset")
        return needs

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        t = self.spec.tensors
        self.in_weight, _ = stacked_rows([tensors[t["x"]], tensors[t["y"]]])
        self.o = tensors[t["o"]].contiguous()
        self.gates = torch.cat([tensors[t["ra"]], tensors[t["ri"]]], dim=1).contiguous()   # [blocks, 2 * block, block]
        self.conv = tensors[t["conv"]].float().t().contiguous()                            # [taps, width]
        for name in ("x_bias", "y_bias", "conv_bias", "ra_bias", "ri_bias"):
            setattr(self, name, tensors[t[name]].float().reshape(-1).contiguous())
        lam = tensors[t["lam"]].double()
        self.decay = (-self.decay_scale * torch.logaddexp(lam, torch.zeros_like(lam))).float().contiguous()

    def cache_need(self) -> StateNeed:
        return StateNeed((self.width,), dtype="float32")

    def bind_cache(self, binding) -> None:
        self.states = binding.states

    def state_holders(self) -> list:
        """What else keeps something per request for this mixer: the convolution's inputs."""
        return [self.ring]

    def captures_state_steps(self) -> bool:
        return True

    def plan_key(self):
        return SEQUENCE_ROWS_KEY

    def plan_step(self, step) -> dict:
        return sequence_rows_plan(step)

    def projections(self) -> torch.Tensor:
        """The operand of this mixer's projections of its input, [rows, H]: x, then y."""
        return self.in_weight

    def _gate_products(self, u: torch.Tensor) -> torch.Tensor:
        """fp32 [blocks, T, 2 * block]: every block's Ra u and Ri u, unrounded."""
        tokens = u.shape[0]
        if u.dtype == torch.bfloat16:
            parts = u.view(tokens, self.blocks, self.block).transpose(0, 1)
            return torch.bmm(parts, self.gates.transpose(1, 2), out_dtype=torch.float32)
        pre = torch.empty((self.blocks, tokens, 2 * self.block), dtype=torch.float32, device=u.device)
        for b in range(self.blocks):
            ops.gemm_f32(u[:, b * self.block:(b + 1) * self.block], self.gates[b], pre[b])
        return pre

    def forward_columns(self, proj: torch.Tensor, row_stride: int, h: torch.Tensor, batch, bias_taken: bool) -> torch.Tensor:
        """The mixer from its projections: proj [T, channels], columns of a matrix whose rows are `row_stride` apart."""
        tokens = proj.shape[0]
        x, y = proj[:, :self.width], proj[:, self.column:self.column + self.width]
        ring = self.ring.binding.states
        out = torch.empty((tokens, self.width), dtype=proj.dtype, device=proj.device)
        if proj.dtype == torch.bfloat16 and int(batch.n_decode) == tokens:
            ops.linear_step(x, row_stride, self.x_bias, self.conv, self.conv_bias, ring, self.gates, self.ra_bias,
                            self.ri_bias, self.decay, y, self.y_bias, self.states, batch.entry, batch.slots, batch.pos, out)
            return linear(out, self.o)
        plan = batch.plans[SEQUENCE_ROWS_KEY]
        u = torch.empty((tokens, self.width), dtype=proj.dtype, device=proj.device)
        ops.ring_conv(x, row_stride, self.x_bias, self.conv, self.conv_bias, ring, plan["first"], batch.entry, batch.slots,
                      batch.pos, u)
        ops.linear_scan(self._gate_products(u), self.ra_bias, self.ri_bias, self.decay, u, y, self.y_bias, x, row_stride,
                        ring, self.states, plan["first"], plan["count"], batch.slots, batch.pos,
                        max(batch.host_query_lens, default=1), out)
        return linear(out, self.o)

    def forward(self, h: torch.Tensor, batch) -> torch.Tensor:
        proj = linear(h, self.in_weight)
        return self.forward_columns(proj, proj.stride(0), h, batch, False)
