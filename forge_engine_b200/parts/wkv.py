"""Time mixing with a matrix state per head whose decay depends on the token, per key channel.

Five projections r, k, v, g, w read five mixes h + (h' - h) mu_s of the token's normalised row h
and the row before it, h'.  With w = exp(-exp(A tanh(B mix_w) + base)) per head and key channel,
o_t = (S + diag(u) k v^T)^T r and then S <- diag(w) S + k v^T; each head's o is divided by its root
mean square, the heads are weighted, multiplied by silu(g) and projected.

The mixer makes its own input (``enter``): residual sum, norm and mixes are taken in 32-bit and
rounded once - in one launch where every entry brings one token - together with the rounded row a
feed-forward beside it reads.  r, k, v and g are one grouped product over the four mixes; their 32-bit
sums, the decays and the state stay 32-bit.  A request keeps the state S and its last row h.
"""

from __future__ import annotations

import torch

from ..cache.manager import CacheNeeds, StateSpec
from ..config.specs import local_name
from ..errors import ConfigError
from ..ops import native
from .base import BuildContext, CacheView, Mixer, WeightInfo, register_part
from .linear import Linear, fused_rows

MIXES = ("r", "k", "v", "g", "w")


class WKV(Mixer):
    graph_safe = True      # the states are indexed on the device, by the batch's slots

    def __init__(self, spec, weights: dict, ctx: BuildContext) -> None:
        self.spec, self.ctx = spec, ctx
        self.h, self.d, self.width = spec.num_heads, spec.head_dim, spec.hidden_size
        self.size = self.h * self.d
        name = lambda canonical: local_name(spec, canonical)  # noqa: E731
        vector = lambda key: weights[name(key)].to(device=ctx.device, dtype=torch.float32).reshape(-1)  # noqa: E731
        self.mu = torch.stack([vector(f"mu.{s}") for s in MIXES]).contiguous()
        self.proj = fused_rows(weights, [name(s) for s in MIXES[:4]], [self.size] * 4).view(4, self.size, self.width)
        self.low = Linear(weights[name("w1")], status=ctx.status)
        self.up = weights[name("w2")].to(device=ctx.device, dtype=torch.float32).t().contiguous()     # [rank, channels]
        self.base, self.bonus, self.norm = (vector(key).contiguous() for key in ("w0", "u", "norm"))
        self.o_proj = Linear(weights[name("o")], status=ctx.status)
        self._plans: dict = {}

    @classmethod
    def weight_shapes(cls, spec) -> dict:
        name = lambda canonical: local_name(spec, canonical)  # noqa: E731
        w, size = spec.hidden_size, spec.num_heads * spec.head_dim
        shapes = {name(f"mu.{s}"): WeightInfo((w,), "small") for s in MIXES}
        shapes.update({name(s): WeightInfo((size, w)) for s in MIXES[:4]})
        shapes.update({
            # rank None: the stored tensors say how many rows the decay's two matrices share
            name("w1"): WeightInfo((spec.rank, w)),
            name("w2"): WeightInfo((size, spec.rank)),
            name("w0"): WeightInfo((size,), "bias"),
            name("u"): WeightInfo((spec.num_heads, spec.head_dim), "bias"),
            name("norm"): WeightInfo((size,), "norm"),
            name("o"): WeightInfo((w, size)),
        })
        return shapes

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(state=StateSpec((self.h, self.d, self.d), "float32"),
                          states=(("previous", StateSpec((self.width,), "float32")),))

    def enter(self, h, pending, shift, norm, batch, cache: CacheView, plain: bool):
        """Adds ``pending`` and ``shift`` into the stream, normalises it and returns (the mixes
        [5, N, width], the normalised rows in the activation dtype or None)."""
        if getattr(norm, "stream_kind", None) != native.NORM_RMS:
            raise ConfigError("time mixing reads an RMS norm's rows")
        n = h.shape[0]
        mixed = torch.empty((len(MIXES), n, self.width), dtype=self.ctx.dtype, device=h.device)
        rows = torch.empty((n, self.width), dtype=self.ctx.dtype, device=h.device) if plain else None
        state = cache.states["previous"]
        if batch.max_new == 1 and batch.n_entries == n:
            native.token_shift(self.mu, state, batch.slots, batch.cu_tokens, batch.token_entry, mixed, rows, residual=h,
                               update=pending, shift=shift, weight=norm.weight, eps=norm.eps)
        else:
            y = torch.empty((n, self.width), dtype=torch.float32, device=h.device)
            native.add_rmsnorm(h, pending, norm.weight, y, norm.eps, shift=shift)
            native.token_shift(self.mu, state, batch.slots, batch.cu_tokens, batch.token_entry, mixed, rows, y=y)
        return mixed, rows

    def _grouped_plan(self, n: int, device) -> dict:
        """Where the four products' rows lie, for the grouped tcgen05 product: one row tile each."""
        plan = self._plans.get(n)
        if plan is None:
            table = torch.tensor([0, 1, 2, 3] + [i * n for i in range(4)] + [i * n for i in range(5)], dtype=torch.int32).to(device)
            plan = self._plans[n] = {"tile_expert": table[:4], "tile_row": table[4:8], "offsets": table[8:]}
        return plan

    def _project(self, mixed):
        """r, k, v, g [4, N, heads * dim] as 32-bit sums."""
        n, x = mixed.shape[1], mixed[:4]
        bf16 = x.dtype == torch.bfloat16 and self.proj.dtype == torch.bfloat16
        if bf16 and n > native.TC5_MAX_ROWS:
            return torch.bmm(x, self.proj.transpose(1, 2), out_dtype=torch.float32)
        out = torch.empty((4, n, self.size), dtype=torch.float32, device=x.device)
        if bf16 and self.width % 8 == 0:
            native.gemm_tc5_grouped(x.reshape(4 * n, self.width), self.proj, out.view(4 * n, self.size), native.TC5_STORE_F32,
                                    self._grouped_plan(n, x.device), native.tc5_tile(n), 4, self.ctx.status)
        else:
            native.gemm_simt_batched(x.transpose(0, 1), self.proj, out.transpose(0, 1))
        return out

    def forward(self, mixed, batch, cache: CacheView):
        n = mixed.shape[1]
        with self.ctx.section("mixer.projection"):
            r, k, v, g = self._project(mixed)
            low = self.low(mixed[4], out_dtype=torch.float32)
            decay = torch.empty((n, self.size), dtype=torch.float32, device=mixed.device)
            native.wkv_decay(low, self.up, self.base, decay)
        heads = torch.empty((n, self.size), dtype=self.ctx.dtype, device=mixed.device)
        with self.ctx.section("mixer.recurrence"):
            native.wkv(r, k, v, decay, self.bonus, self.norm, g, self.spec.norm_eps, cache.state, batch.slots, batch.cu_tokens,
                       heads, batch.n_entries, batch.max_new, self.ctx.status)
        with self.ctx.section("mixer.o_proj"):
            return self.o_proj(heads, out_dtype=torch.float32)


register_part("wkv", WKV, replace=True)
