"""Two mixers that read the same input, joined as half the sum of their normalised outputs:
y = 1/2 (left / rms(left) * w_left + right / rms(right) * w_right), the root mean squares over the
model's width, or (``scales``) as a weighted sum a left + b right.  The mixers' last projections
leave 32-bit sums; joining them is one kernel.  What the two keep between steps is kept side by side: one of them may keep keys and values,
one may keep states."""

from __future__ import annotations

from collections.abc import Mapping

import torch

from ..cache.manager import CacheNeeds
from ..config.specs import local_name
from ..errors import ConfigError
from ..ops import native
from .base import BuildContext, CacheView, Mixer, WeightInfo, build_part, part_class, register_part, summed_update

SIDES = ("left", "right")


class _Side(Mapping):
    """The tensors under ``<prefix>.`` by the names behind it, looked up when asked for."""

    def __init__(self, weights, prefix: str) -> None:
        self._weights, self._prefix = weights, prefix + "."

    def __getitem__(self, local: str):
        return self._weights[self._prefix + local]

    def __iter__(self):
        return (name[len(self._prefix):] for name in self._weights if name.startswith(self._prefix))

    def __len__(self) -> int:
        return sum(1 for _ in self)


class SideBySide(Mixer):
    def __init__(self, spec, weights: dict, ctx: BuildContext) -> None:
        self.spec, self.ctx = spec, ctx
        self.sides = [build_part(getattr(spec, side), _Side(weights, side), ctx) for side in SIDES]
        self.scales = None if getattr(spec, "scales", None) is None else tuple(float(s) for s in spec.scales)
        self.norms = [] if self.scales is not None else [weights[local_name(spec, f"{side}.out")].to(device=ctx.device, dtype=torch.float32).contiguous() for side in SIDES]
        self.cache_needs()      # refuses two mixers that want the same place

    @classmethod
    def weight_shapes(cls, spec) -> dict:
        shapes = {}
        for side in SIDES:
            inner = getattr(spec, side)
            shapes.update({f"{side}.{name}": info for name, info in part_class(inner).weight_shapes(inner).items()})
            if getattr(spec, "scales", None) is None:
                shapes[local_name(spec, f"{side}.out")] = WeightInfo((spec.hidden_size,), "norm")
        return shapes

    @property
    def graph_safe(self) -> bool:
        return all(getattr(side, "graph_safe", False) for side in self.sides)

    def plan_step(self, entries: list, page_size: int, plans: dict) -> None:
        for side in self.sides:
            planner = getattr(side, "plan_step", None)
            if planner is not None:
                planner(entries, page_size, plans)

    def cache_needs(self) -> CacheNeeds:
        needs = [side.cache_needs() for side in self.sides]
        pick = {}
        for key in ("kv", "state", "own_state"):
            given = [getattr(need, key) for need in needs if getattr(need, key) is not None]
            if len(given) > 1:
                raise ConfigError(f"two mixers side by side that both keep {key!r} are not implemented")
            pick[key] = given[0] if given else None
        names = [name for need in needs for name, _ in need.states]
        if len(set(names)) != len(names):
            raise ConfigError(f"two mixers side by side keep states of the same name: {names}")
        return CacheNeeds(**pick, states=tuple(state for need in needs for state in need.states))

    def _update(self, side, x, batch, cache: CacheView):
        """A side's update, as the 32-bit sums of its output projection where it has one."""
        return summed_update(self.ctx, side, x, batch, cache).float()

    def forward(self, x, batch, cache: CacheView):
        left, right = (self._update(side, x, batch, cache) for side in self.sides)
        out = torch.empty_like(left)
        with self.ctx.section("mixer.join"):
            if self.scales is not None:
                native.weighted_sum(left, right, self.scales[0], self.scales[1], out)
                return out
            native.norm_pair(left, right, self.norms[0], self.norms[1], out, self.spec.norm_eps, 0.5)
        return out


register_part("side_by_side", SideBySide, replace=True)
