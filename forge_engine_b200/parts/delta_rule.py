"""The gated delta rule: a matrix state per head that is decayed and then corrected towards the
value of every key.

q and k [kv_heads x dim] (shared by groups of heads) and v [heads x vdim] pass a short causal
convolution over time and silu; q and k are unit vectors per head, q times dim^(-1/2).  With beta =
sigmoid(W_b x) and g = exp(-exp(A_log) softplus(W_a x + dt_bias)) per head: S <- g S; u = beta
(v - S^T k); S <- S + k u^T; o = S^T q.  Each head's o is divided by its root mean square, weighted,
multiplied by silu(W_g x) and projected.

One fused projection gives q, k, v, the output gate and both gates' logits as 32-bit sums; one kernel
takes convolution, activation, unit vectors and gates; the recurrence and its norm follow in 32-bit.
A request keeps the state S and the convolution's last taps - 1 inputs.
"""

from __future__ import annotations

import torch

from ..cache.manager import CacheNeeds, StateSpec
from ..config.specs import local_name
from ..errors import ConfigError
from ..ops import native
from .base import BuildContext, CacheView, Mixer, WeightInfo, register_part
from .linear import Linear, fused_rows


class DeltaRule(Mixer):
    graph_safe = True      # the states are indexed on the device, by the batch's slots

    def __init__(self, spec, weights: dict, ctx: BuildContext) -> None:
        if spec.num_heads % spec.num_kv_heads:
            raise ConfigError("num_heads must be a multiple of num_kv_heads")
        self.spec, self.ctx = spec, ctx
        self.h, self.kvh, self.dk, self.dv, self.taps = spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.v_head_dim, spec.taps
        name = lambda canonical: local_name(spec, canonical)  # noqa: E731
        qk, v = self.kvh * self.dk, self.h * self.dv
        self.channels = 2 * qk + v
        rows = [qk, qk, v, v, self.h, self.h]
        self.proj = Linear(fused_rows(weights, [name(s) for s in ("q", "k", "v", "g", "b", "a")], rows), status=ctx.status)
        conv = fused_rows(weights, [name(f"{s}.conv") for s in ("q", "k", "v")], [qk, qk, v])
        # stored [channels, taps]; the kernel reads a tap's weights side by side
        self.conv = conv.to(device=ctx.device, dtype=torch.float32).t().contiguous()
        vector = lambda key: weights[name(key)].to(device=ctx.device, dtype=torch.float32).reshape(-1).contiguous()  # noqa: E731
        self.a_log, self.dt_bias, self.norm = vector("A_log"), vector("dt_bias"), vector("norm")
        self.o_proj = Linear(weights[name("o")], status=ctx.status)

    @classmethod
    def weight_shapes(cls, spec) -> dict:
        name = lambda canonical: local_name(spec, canonical)  # noqa: E731
        w, h = spec.hidden_size, spec.num_heads
        qk, v = spec.num_kv_heads * spec.head_dim, h * spec.v_head_dim
        shapes = {}
        for s, rows in (("q", qk), ("k", qk), ("v", v)):
            shapes[name(s)] = WeightInfo((rows, w))
            shapes[name(f"{s}.conv")] = WeightInfo((rows, spec.taps), "norm")
        shapes.update({
            name("g"): WeightInfo((v, w)),
            name("b"): WeightInfo((h, w)),
            name("a"): WeightInfo((h, w)),
            name("A_log"): WeightInfo((h,), "bias"),
            name("dt_bias"): WeightInfo((h,), "bias"),
            name("norm"): WeightInfo((spec.v_head_dim,), "norm"),
            name("o"): WeightInfo((w, v)),
        })
        return shapes

    def cache_needs(self) -> CacheNeeds:
        states = (("conv", StateSpec((self.taps - 1, self.channels), "float32")),) if self.taps > 1 else ()
        return CacheNeeds(state=StateSpec((self.h, self.dk, self.dv), "float32"), states=states)

    def forward(self, x, batch, cache: CacheView):
        n, v = x.shape[0], self.h * self.dv
        with self.ctx.section("mixer.projection"):
            proj = self.proj(x, out_dtype=torch.float32)
        heads = torch.empty((n, v), dtype=self.ctx.dtype, device=x.device)
        with self.ctx.section("mixer.recurrence"):
            qkv = torch.empty((n, self.channels), dtype=torch.float32, device=x.device)
            gates = torch.empty((n, self.h, 2), dtype=torch.float32, device=x.device)
            native.delta_prepare(proj, self.channels + v, self.channels + v + self.h, self.conv, cache.states.get("conv"),
                                 batch.slots, batch.cu_tokens, batch.token_entry, self.a_log, self.dt_bias, self.kvh, self.dk, self.h,
                                 self.dv, qkv, gates, batch.n_entries)
            native.delta_rule(qkv, gates, proj[:, self.channels :], self.norm, self.spec.norm_eps, cache.state, batch.slots,
                              batch.cu_tokens, heads, self.kvh, batch.n_entries, batch.max_new, self.ctx.status)
        with self.ctx.section("mixer.o_proj"):
            return self.o_proj(heads, out_dtype=torch.float32)


register_part("delta_rule", DeltaRule, replace=True)
