"""A matrix memory with exponential gates and a normaliser per head.

Log gates i = c tanh((W_i x + b_i) / c) and f = logsigmoid(c tanh((W_f x + b_f) / c)); with the running
maximum m_t = max(f + m_(t-1), i), zero at the start, S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t)
k v^T, the normaliser n likewise with k alone, and o = S^T q / (max(|n . q|, e^(-m_t)) + 1e-6), q
times dim^(-1/2).  Each head's o is divided by its root mean square, the heads are weighted,
multiplied by sigmoid(W_g x) and projected.

One fused projection gives everything as 32-bit sums; gates, recurrence and norm are one kernel (for
prompt portions: a few, chunk by chunk).  A request keeps S, n and m, all 32-bit.
"""

from __future__ import annotations

import torch

from ..cache.manager import CacheNeeds, StateSpec
from ..config.specs import local_name
from ..errors import ConfigError
from ..ops import native
from .base import BuildContext, CacheView, Mixer, WeightInfo, register_part
from .linear import Linear, fused_rows


class MatrixMemory(Mixer):
    graph_safe = True      # the states are indexed on the device, by the batch's slots

    def __init__(self, spec, weights: dict, ctx: BuildContext) -> None:
        if not spec.gate_cap > 0:
            raise ConfigError("gate_cap must be positive")
        self.spec, self.ctx = spec, ctx
        self.h, self.dk, self.dv = spec.num_heads, spec.head_dim, spec.v_head_dim
        name = lambda canonical: local_name(spec, canonical)  # noqa: E731
        qk, v = self.h * self.dk, self.h * self.dv
        rows = [qk, qk, v, v, self.h, self.h]
        self.proj = Linear(fused_rows(weights, [name(s) for s in ("q", "k", "v", "g", "i", "f")], rows), status=ctx.status)
        self.offsets = tuple(sum(rows[:j]) for j in range(len(rows)))
        vector = lambda key: weights[name(key)].to(device=ctx.device, dtype=torch.float32).reshape(-1).contiguous()  # noqa: E731
        self.i_bias, self.f_bias, self.norm = vector("i.b"), vector("f.b"), vector("norm")
        self.o_proj = Linear(weights[name("o")], status=ctx.status)

    @classmethod
    def weight_shapes(cls, spec) -> dict:
        name = lambda canonical: local_name(spec, canonical)  # noqa: E731
        w, h = spec.hidden_size, spec.num_heads
        qk, v = h * spec.head_dim, h * spec.v_head_dim
        return {
            name("q"): WeightInfo((qk, w)),
            name("k"): WeightInfo((qk, w)),
            name("v"): WeightInfo((v, w)),
            name("g"): WeightInfo((v, w)),
            name("i"): WeightInfo((h, w)),
            name("f"): WeightInfo((h, w)),
            name("i.b"): WeightInfo((h,), "bias"),
            name("f.b"): WeightInfo((h,), "bias"),
            name("norm"): WeightInfo((v,), "norm"),
            name("o"): WeightInfo((w, v)),
        }

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(state=StateSpec((self.h, self.dk, self.dv), "float32"),
                          states=(("normaliser", StateSpec((self.h, self.dk), "float32")), ("top", StateSpec((self.h,), "float32"))))

    def attend(self, x, batch, cache: CacheView):
        """Everything but the output projection: the normalised, gated heads [N, heads * vdim]."""
        with self.ctx.section("mixer.projection"):
            proj = self.proj(x, out_dtype=torch.float32)
        heads = torch.empty((x.shape[0], self.h * self.dv), dtype=self.ctx.dtype, device=x.device)
        with self.ctx.section("mixer.recurrence"):
            native.matrix_memory(proj, self.offsets, self.i_bias, self.f_bias, self.spec.gate_cap, self.dk ** -0.5, self.norm,
                                 self.spec.norm_eps, cache.state, cache.states["normaliser"], cache.states["top"], batch.slots,
                                 batch.cu_tokens, heads, batch.n_entries, batch.max_new, self.ctx.status)
        return heads

    def forward(self, x, batch, cache: CacheView):
        heads = self.attend(x, batch, cache)
        with self.ctx.section("mixer.o_proj"):
            return self.o_proj(heads, out_dtype=torch.float32)


register_part("matrix_memory", MatrixMemory, replace=True)
