"""Griffin's recurrent block around a real-gated linear recurrent unit.

y = gelu_tanh(W_y x + b) and u = conv(W_x x + b), a causal convolution over time with a few taps and a
bias per channel.  The channels fall into equal parts; in each r = sigmoid(R u + b), i = sigmoid(I u + b);
log a = -strength r softplus(lam); S_t = a S_(t-1) + sqrt(1 - a^2) i u_t per channel, zero at the start;
the update is W_o (S y).

One fused projection gives y and x as 32-bit sums (their biases are added by the kernels that read them);
convolution, both gate products, recurrence and gate
are one kernel where every entry brings one token, else three (tiles of tokens side by side, their states
chained, the outputs).  A request keeps S and the convolution's last taps - 1 inputs, 32-bit.
"""

from __future__ import annotations

import torch

from ..cache.manager import CacheNeeds, StateSpec
from ..config.specs import local_name
from ..errors import ConfigError
from ..ops import native
from .base import BuildContext, CacheView, Mixer, WeightInfo, register_part
from .linear import Linear, fused_rows


class RGLRU(Mixer):
    graph_safe = True      # the states are indexed on the device, by the batch's slots

    def __init__(self, spec, weights: dict, ctx: BuildContext) -> None:
        if spec.width % spec.blocks:
            raise ConfigError("width must be a multiple of blocks")
        self.spec, self.ctx = spec, ctx
        self.width, self.taps = spec.width, spec.taps
        name = lambda canonical: local_name(spec, canonical)  # noqa: E731
        rows = [self.width, self.width]
        self.proj = Linear(fused_rows(weights, [name("y"), name("x")], rows), status=ctx.status)
        vector = lambda key: weights[name(key)].to(device=ctx.device, dtype=torch.float32).reshape(-1).contiguous()  # noqa: E731
        # stored [channels, taps]; the kernels read a tap's weights side by side
        self.conv = weights[name("conv")].to(device=ctx.device, dtype=torch.float32).t().contiguous()
        self.y_bias, self.x_bias, self.conv_bias = vector("y.b"), vector("x.b"), vector("conv.b")
        self.r_bias, self.i_bias = vector("ra.b"), vector("ri.b")
        self.r_weight, self.i_weight = weights[name("ra")].contiguous(), weights[name("ri")].contiguous()
        if self.r_weight.dtype != self.i_weight.dtype:
            self.r_weight, self.i_weight = self.r_weight.float(), self.i_weight.float()
        # log a = rate r: softplus in 64-bit, rounded once
        lam = weights[name("lam")].double().reshape(-1)
        softplus = lam.clamp(min=0) + torch.log1p(torch.exp(-lam.abs()))
        self.rate = (-float(spec.strength) * softplus).float().to(ctx.device).contiguous()
        self.o_proj = Linear(weights[name("o")], status=ctx.status)

    @classmethod
    def weight_shapes(cls, spec) -> dict:
        name = lambda canonical: local_name(spec, canonical)  # noqa: E731
        w, c, part = spec.hidden_size, spec.width, spec.width // spec.blocks
        shapes = {}
        for s in ("y", "x"):
            shapes[name(s)] = WeightInfo((c, w))
            shapes[name(f"{s}.b")] = WeightInfo((c,), "bias")
        for s in ("ra", "ri"):
            shapes[name(s)] = WeightInfo((spec.blocks, part, part))
            shapes[name(f"{s}.b")] = WeightInfo((spec.blocks, part), "bias")
        shapes.update({
            name("conv"): WeightInfo((c, spec.taps), "small"),
            name("conv.b"): WeightInfo((c,), "bias"),
            name("lam"): WeightInfo((c,), "bias"),
            name("o"): WeightInfo((w, c)),
        })
        return shapes

    def cache_needs(self) -> CacheNeeds:
        states = (("conv", StateSpec((self.taps - 1, self.width), "float32")),) if self.taps > 1 else ()
        return CacheNeeds(state=StateSpec((self.width,), "float32"), states=states)

    def attend(self, x, batch, cache: CacheView):
        """Everything but the output projection: S y [N, width]."""
        with self.ctx.section("mixer.projection"):
            proj = self.proj.sums(x)
        out = torch.empty((x.shape[0], self.width), dtype=self.ctx.dtype, device=x.device)
        with self.ctx.section("mixer.recurrence"):
            native.rglru(proj, 0, self.width, self.conv, self.conv_bias, self.r_weight, self.i_weight, self.y_bias, self.x_bias,
                         self.r_bias, self.i_bias, self.rate, cache.state, cache.states.get("conv"), batch.slots, batch.cu_tokens, batch.token_entry, out,
                         batch.n_entries, batch.max_new, self.ctx.status)
        return out

    def forward(self, x, batch, cache: CacheView):
        out = self.attend(x, batch, cache)
        with self.ctx.section("mixer.o_proj"):
            return self.o_proj(out, out_dtype=torch.float32)


register_part("rglru", RGLRU, replace=True)
