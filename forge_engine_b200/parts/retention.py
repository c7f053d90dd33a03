"""Retention: linear attention with a fixed decay per head on rotated queries and keys.

q = W_q x, k = W_k x [heads x dim], both rotated by position, v = W_v x [heads x vdim]; per head
S_t = decay_h S_(t-1) + c k_t v_t^T, o_t = S_t^T q_t.  Each head's o is divided by its root mean square
(optionally weighted), multiplied by silu(W_g x) and projected.

One fused projection gives q, k, v and the gate as 32-bit sums; rotation, recurrence, norm and gate are
one kernel (for prompt portions: a few, chunk by chunk, after a launch that rotates q and k in place).
A request keeps S, 32-bit.
"""

from __future__ import annotations

import torch

from ..cache.manager import CacheNeeds, StateSpec
from ..config.specs import local_name
from ..errors import ConfigError
from ..ops import native
from .base import BuildContext, CacheView, Mixer, WeightInfo, build_part, register_part
from .linear import Linear, fused_rows


class Retention(Mixer):
    @property
    def graph_safe(self) -> bool:
        """The state is indexed on the device, by the batch's slots; the position encoding decides for itself."""
        return bool(getattr(self.position, "graph_safe", False))

    def __init__(self, spec, weights: dict, ctx: BuildContext) -> None:
        if len(spec.decay) != spec.num_heads or not all(0.0 <= float(d) <= 1.0 for d in spec.decay):
            raise ConfigError("one decay between 0 and 1 per head is needed")
        self.spec, self.ctx = spec, ctx
        self.h, self.dk, self.dv = spec.num_heads, spec.head_dim, spec.v_head_dim
        name = lambda canonical: local_name(spec, canonical)  # noqa: E731
        qk, v = self.h * self.dk, self.h * self.dv
        rows = [qk, qk, v, v]
        self.proj = Linear(fused_rows(weights, [name(s) for s in ("q", "k", "v", "g")], rows), status=ctx.status)
        self.offsets = tuple(sum(rows[:j]) for j in range(len(rows)))
        self.norm = weights[name("norm")].to(device=ctx.device, dtype=torch.float32).contiguous() if spec.norm_weight else None
        self.o_proj = Linear(weights[name("o")], status=ctx.status)
        self.decay = torch.tensor(spec.decay, dtype=torch.float64).float().to(ctx.device)
        self.position = build_part(spec.position, {}, ctx)
        self.rot = 0 if self.position.rotary() is None else int(self.position.rotary()[1])

    @classmethod
    def weight_shapes(cls, spec) -> dict:
        name = lambda canonical: local_name(spec, canonical)  # noqa: E731
        qk, v, w = spec.num_heads * spec.head_dim, spec.num_heads * spec.v_head_dim, spec.hidden_size
        shapes = {name("q"): WeightInfo((qk, w)), name("k"): WeightInfo((qk, w)), name("v"): WeightInfo((v, w)),
                  name("g"): WeightInfo((v, w)), name("o"): WeightInfo((w, v))}
        if spec.norm_weight:
            shapes[name("norm")] = WeightInfo((spec.v_head_dim,), "norm")
        return shapes

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(state=StateSpec((self.h, self.dk, self.dv), "float32"))

    def attend(self, x, batch, cache: CacheView):
        """Everything but the output projection: the heads' outputs [N, heads * v_head_dim]."""
        with self.ctx.section("mixer.projection"):
            proj = self.proj(x, out_dtype=torch.float32)
        heads = torch.empty((x.shape[0], self.h * self.dv), dtype=self.ctx.dtype, device=x.device)
        with self.ctx.section("mixer.recurrence"):
            table = self.position.table(batch) if self.rot else None
            interleaved = bool(getattr(self.position, "interleaved", False))
            if table is not None and batch.max_new >= native.state_long_from():
                # q and k lie side by side: 2 x heads rows of dim, rotated where they are
                qk = proj[:, : 2 * self.h * self.dk]
                native.qkv_prepare(q=qk, q_heads=2 * self.h, q_dim=self.dk, q_out=qk, q_out_strides=(proj.shape[1], self.dk),
                                   table=table, rot_dims=self.rot, interleaved=interleaved, positions=batch.positions,
                                   token_entry=batch.token_entry, status=self.ctx.status)
                table = None
            native.retention(proj, self.offsets, float(self.spec.key_scale), self.decay, table, self.rot, interleaved, self.norm,
                             self.spec.norm_eps, cache.state, batch.slots, batch.cu_tokens, heads, batch.n_entries, batch.max_new,
                             self.ctx.status)
        return heads

    def forward(self, x, batch, cache: CacheView):
        heads = self.attend(x, batch, cache)
        with self.ctx.section("mixer.o_proj"):
            return self.o_proj(heads, out_dtype=torch.float32)


register_part("retention", Retention, replace=True)
