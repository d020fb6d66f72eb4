"""A matrix memory with exponential gates (the mLSTM recurrence): a recurrent mixer with a matrix state, a normaliser
and a stabiliser per head."""

from __future__ import annotations

import numpy as np
import torch

from ..kernels import ops
from .filtered_attention import stacked_rows
from .linear import linear
from .registry import BuildContext, Part, register_part
from .spec import PartSpec, StateNeed, TensorNeed


@register_part("mixer", "matrix_memory")
class MatrixMemory(Part):
    """Per head a state S [dim, vdim], a normaliser n [dim] and a stabiliser m, fp32, zero at a sequence's start and
    carried from token to token:

        q, k = Wq h * dim^(-1/2), Wk h   [heads, dim];   v = Wv h   [heads, vdim]
        i = cap tanh((Wi h + bi) / cap);   f = logsigmoid(cap tanh((Wf h + bf) / cap))       one each per head
        m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T;  n likewise with k alone;  m <- m'
        o = S^T q / (max(|n . q|, exp(-m)) + 1e-6)
        out = Wo (o / sqrt(mean(o^2) + eps) * norm * sigmoid(Wg h))

    q, k, v and g are one product; the gate logits are fp32 throughout. float32 engine, and shapes the other kernels do
    not take: one kernel walks each entry's tokens. bfloat16: prompt portions in chunks on tensor cores, leading single
    tokens in one launch that forms the gate logits itself (csrc/matrix_memory.cu).

    params: hidden_size, n_heads, head_dim (dim), value_dim (vdim), gate_cap, eps. tensors: q, k [nh*dim, H], v, g
    [nh*vdim, H], i, f [nh, H], i_bias, f_bias [nh], norm [nh*vdim], o [H, nh*vdim]."""

    def __init__(self, spec: PartSpec, ctx: BuildContext):
        super().__init__(spec, ctx)
        self.hidden = int(self.param("hidden_size"))
        self.n_heads = int(self.param("n_heads"))
        self.dim = int(self.param("head_dim"))
        self.vdim = int(self.param("value_dim"))
        self.cap = float(self.param("gate_cap"))
        self.eps = float(self.param("eps"))
        if self.cap <= 0.0:
            raise ValueError(f"matrix_memory: gate_cap must be positive, got {self.cap}")
        self.stacked = self.gates = self.o = self.norm = None
        self.starts: list[int] = []
        self.gate_bias: tuple = ()
        self.states = None
        self._forms: tuple[bool, bool] | None = None

    @classmethod
    def tensor_needs(cls, spec: PartSpec) -> dict[str, TensorNeed]:
        p, t = spec.params, spec.tensors
        h, nh, hd, vd = (int(p[k]) for k in ("hidden_size", "n_heads", "head_dim", "value_dim"))
        return {t["q"]: TensorNeed((nh * hd, h)), t["k"]: TensorNeed((nh * hd, h)), t["v"]: TensorNeed((nh * vd, h)),
                t["g"]: TensorNeed((nh * vd, h)), t["i"]: TensorNeed((nh, h)), t["f"]: TensorNeed((nh, h)),
                t["i_bias"]: TensorNeed((nh,), role="offset"), t["f_bias"]: TensorNeed((nh,), role="offset"),
                t["norm"]: TensorNeed((nh * vd,), role="vector"), t["o"]: TensorNeed((h, nh * vd))}

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        t = self.spec.tensors
        self.stacked, self.starts = stacked_rows([tensors[t[name]] for name in ("q", "k", "v", "g")])
        self.gates = torch.cat([tensors[t["i"]], tensors[t["f"]]], dim=0).contiguous()
        self.gate_bias = tuple(tensors[t[name]].float().contiguous() for name in ("i_bias", "f_bias"))
        self.norm = tensors[t["norm"]].float().contiguous()
        self.o = tensors[t["o"]].contiguous()

    def cache_need(self) -> StateNeed:
        return StateNeed((self.n_heads, ops.matrix_memory_head_floats(self.dim, self.vdim)), dtype="float32")

    def bind_cache(self, binding) -> None:
        self.states = binding.states

    def captures_state_steps(self) -> bool:
        return True

    def forms(self) -> tuple[bool, bool]:
        """Whether this layer's portions go in chunks, and its single tokens through the one-launch kernel."""
        if self._forms is None:
            dtype = self.ctx.dtype
            self._forms = (ops.matrix_memory_chunks_supports(self.dim, self.vdim, dtype),
                           ops.matrix_memory_step_supports(self.dim, self.vdim, self.hidden, dtype))
        return self._forms

    def plan_key(self):
        return ("matrix memory",)

    def plan_step(self, step) -> dict:
        """For the walk: every entry's first row and row count. For the chunked form: the chunks of the entries that
        bring more than one token (they follow those that bring one), and each such entry's run of chunks."""
        plan = {"first": np.asarray(step.first_rows, dtype=np.int32), "count": np.asarray(step.query_lens, dtype=np.int32),
                "chunks": None, "spans": None}
        if self.ctx.dtype != torch.bfloat16 or step.n_decode == step.n_entries:
            return plan
        size = ops.matrix_memory_chunk_tokens()
        chunks, spans = [], []
        for e in range(step.n_decode, step.n_entries):
            n, at = step.query_lens[e], step.first_rows[e]
            spans.append((len(chunks), -(-n // size), e, 0))
            chunks += [(at + r, min(size, n - r), e, int(r + size >= n)) for r in range(0, n, size)]
        plan["chunks"] = np.array(chunks, dtype=np.int32)
        plan["spans"] = np.array(spans, dtype=np.int32)
        return plan

    def forward(self, h: torch.Tensor, batch) -> torch.Tensor:
        tokens = h.shape[0]
        nh, hd, vd = self.n_heads, self.dim, self.vdim
        proj = linear(h, self.stacked)
        columns = tuple(proj[:, at: at + nh * width] for at, width in zip(self.starts, (hd, hd, vd, vd)))
        plan = batch.plans[self.plan_key()]
        out = torch.empty((tokens, nh * vd), dtype=h.dtype, device=h.device)
        in_chunks, in_steps = self.forms()
        single = min(int(batch.n_decode), tokens)
        constants = (self.gate_bias, self.cap, self.norm, self.eps, hd ** -0.5, self.states)
        if (single and not in_steps) or (single < tokens and not in_chunks):
            ops.matrix_memory_walk(columns, proj.stride(0), linear(h, self.gates, out_dtype=torch.float32), *constants,
                                   plan["first"], plan["count"], batch.slots, batch.entry, out, nh, hd, vd)
            return linear(out, self.o)
        if single:
            ops.matrix_memory_step(tuple(c[:single] for c in columns), proj.stride(0), h[:single], self.gates, *constants,
                                   batch.slots, batch.entry[:single], out[:single], nh, hd, vd)
        if single < tokens:
            ops.matrix_memory_chunks(columns, proj.stride(0), linear(h, self.gates, out_dtype=torch.float32), *constants,
                                     batch.slots, plan["chunks"], plan["spans"], out, nh, hd, vd)
        return linear(out, self.o)
