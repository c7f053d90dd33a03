"""The Lofuvik configuration: a decoder whose layers are listed one by one, mixer and feed-forward
of a layer side by side on one norm, a stretch of layers run several times in a row.

``config.json`` names the architecture in ``architecture`` and gives ``vocab``, ``width``,
``norm.eps``, ``layers`` and optionally ``loop``.  Per layer: ``type`` (which mixer), the mixer's
sizes and constants (``mixer``) and its feed-forward (``mlp``, or null).

A layer: with h = norm1(x), x += mixer(h) + ff(h); an RMS norm with a weight.  ``loop``: layers
``start`` .. ``stop`` - 1 run ``times`` times in a row with the same weights and a cache or state per
pass; before each pass but the first the embedding output is added to x once.

Mixers:

* ``wkv`` - time mixing with a matrix state per head and a decay that depends on the token, per
  key channel; every projection reads a mix of the token's row and the one before it;
* ``delta`` - the gated delta rule, q, k and v through a short convolution (``conv`` taps), ``heads``
  value heads over ``kv_heads`` query/key heads;
* ``parallel`` - two mixers on the same input, half the sum of their normalised outputs: ``left``,
  causal grouped-query attention (q and k normalised over the whole projection, the first
  ``rot.dims`` elements of every head rotated, optionally with frequencies scaled by
  ``rot.scaling``: ``factor``, ``original``, ``fast``, ``slow``; scores times ``scale``, capped by
  ``softcap``; a learned sink per head; a sigmoid gate per element of the output), and ``right``, a
  matrix memory with exponential gates capped by ``gate_cap``.

Feed-forward (``mlp.kind`` ``moe``): ``router.experts`` gated SiLU units of which a token uses the
``router.top`` with the largest router logits, weighted by a softmax over those.

Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from dataclasses import dataclass

from ..errors import ConfigError
from .specs import (
    AttentionSpec,
    DeltaRuleSpec,
    GatedMLPSpec,
    LayerSpec,
    MatrixMemorySpec,
    ModelSpec,
    NoPositionSpec,
    NormSpec,
    RotarySpec,
    RoutedMLPSpec,
    RunSpec,
    SideBySideSpec,
    WKVSpec,
)
from .zofadra import _int, _number

MAX_POSITIONS = 1 << 20          # rotary positions have no table; the cache bounds a request first

_BARE = (("weight", ""),)        # a norm's weight is stored under the norm's own name
_ATTENTION = (("q_proj.weight", "q"), ("k_proj.weight", "k"), ("v_proj.weight", "v"), ("o_proj.weight", "o"),
              ("gate_proj.weight", "g"), ("q_norm.weight", "q.norm"), ("k_norm.weight", "k.norm"))
_UNIT = (("gate_proj.weight", "gate"), ("up_proj.weight", "up"), ("down_proj.weight", "down"))
_SCALING = ("factor", "original", "fast", "slow")


@dataclass(frozen=True)
class LofuvikLayer:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass(frozen=True)
class LofuvikLoop:
    start: int
    stop: int
    times: int


def _attention_side(side: dict, where: str) -> dict:
    for key in ("heads", "dim", "vdim"):
        _int(side, key, where)
    if side.get("kv_heads") is None:
        side = dict(side, kv_heads=side["heads"])        # every query head with keys and values of its own
    _int(side, "kv_heads", where)
    if side["heads"] % side["kv_heads"]:
        raise ConfigError(f"{where}.heads must be a multiple of kv_heads")
    _number(side, "scale", where)
    if side.get("softcap") is not None and _number(side, "softcap", where) <= 0:
        raise ConfigError(f"{where}.softcap must be positive")
    rot = side.get("rot")
    if rot is None:
        return side
    if _number(rot, "base", f"{where}.rot") <= 0:
        raise ConfigError(f"{where}.rot.base must be positive")
    dims = _int(rot, "dims", f"{where}.rot", 2)
    if dims % 2 or dims > side["dim"]:
        raise ConfigError(f"{where}.rot.dims={dims} must be even and at most dim={side['dim']}")
    scaling = rot.get("scaling")
    if scaling is not None:
        values = {key: _number(scaling, key, f"{where}.rot.scaling") for key in _SCALING}
        if min(values.values()) <= 0 or rot["base"] == 1:
            raise ConfigError(f"{where}.rot.scaling needs positive numbers and a base other than 1")
    return side


def _check_mixer(kind: str, mixer: dict, where: str) -> dict:
    if kind == "wkv":
        for key in ("heads", "dim"):
            _int(mixer, key, where)
        if mixer.get("rank") is not None:
            _int(mixer, "rank", where)
        return mixer
    if kind == "delta":
        for key in ("heads", "dim", "vdim", "conv"):
            _int(mixer, key, where)
        if mixer.get("kv_heads") is None:
            mixer = dict(mixer, kv_heads=mixer["heads"])
        _int(mixer, "kv_heads", where)
        if mixer["heads"] % mixer["kv_heads"]:
            raise ConfigError(f"{where}.heads must be a multiple of kv_heads")
        return mixer
    left, right = mixer.get("left"), mixer.get("right")
    if not isinstance(left, dict) or not isinstance(right, dict):
        raise ConfigError(f"{where} must have the objects left and right")
    for key in ("heads", "dim", "vdim"):
        _int(right, key, f"{where}.right")
    if _number(right, "gate_cap", f"{where}.right") <= 0:
        raise ConfigError(f"{where}.right.gate_cap must be positive")
    return dict(mixer, left=_attention_side(dict(left), f"{where}.left"), right=dict(right))


@dataclass(frozen=True)
class LofuvikConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple
    loop: LofuvikLoop | None

    architecture = "Lofuvik"

    @classmethod
    def from_dict(cls, raw: dict) -> "LofuvikConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json 'layers' must be a non-empty list")
        eps = _number(raw.get("norm") or {}, "eps", "norm")
        if eps <= 0:
            raise ConfigError("norm.eps must be positive")
        layers = []
        for index, item in enumerate(layers_raw):
            where = f"layers[{index}]"
            kind, mixer = item.get("type"), item.get("mixer")
            if not isinstance(mixer, dict):
                raise ConfigError(f"{where}.mixer must be an object")
            if kind not in ("wkv", "delta", "parallel"):
                raise ConfigError(f"{where}.type={kind!r}; known: wkv, delta, parallel")
            mixer = _check_mixer(kind, dict(mixer), f"{where}.mixer")
            mlp = item.get("mlp")
            if mlp is not None:
                if mlp.get("kind", "moe") != "moe":
                    raise ConfigError(f"{where}.mlp.kind={mlp['kind']!r}; known: moe")
                router = mlp.get("router") or {}
                experts = _int(router, "experts", f"{where}.mlp.router")
                if _int(router, "top", f"{where}.mlp.router") > experts:
                    raise ConfigError(f"{where}.mlp.router.top must be at most experts={experts}")
                _int(mlp.get("expert") or {}, "ff", f"{where}.mlp.expert")
            layers.append(LofuvikLayer(kind, mixer, None if mlp is None else dict(mlp)))
        loop = None
        if raw.get("loop") is not None:
            given = raw["loop"]
            loop = LofuvikLoop(_int(given, "start", "loop", 0), _int(given, "stop", "loop", 0), _int(given, "times", "loop"))
            if not loop.start <= loop.stop <= len(layers):
                raise ConfigError(f"loop: start={loop.start}, stop={loop.stop} do not name a stretch of the {len(layers)} layers")
        return cls(vocab=_int(raw, "vocab", "config"), width=_int(raw, "width", "config"), eps=eps, layers=tuple(layers), loop=loop)

    # ------------------------------------------------------------------------------
    def _norm(self) -> NormSpec:
        return NormSpec(self.width, self.eps, rename=_BARE)

    def _attention_spec(self, m: dict) -> AttentionSpec:
        rot = m.get("rot")
        position = NoPositionSpec()
        if rot is not None:
            scaling = rot.get("scaling")
            position = RotarySpec(head_dim=m["dim"], theta=float(rot["base"]), rotary_dim=int(rot["dims"]), interleaved=False,
                                  exact_frequencies=True,
                                  yarn=None if scaling is None else tuple(float(scaling[key]) for key in _SCALING))
        return AttentionSpec(
            hidden_size=self.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
            qk_norm=True, qk_norm_scope="whole", qk_norm_eps=self.eps, bias=False, scale=float(m["scale"]), position=position,
            softcap=None if m.get("softcap") is None else float(m["softcap"]), sink=True, output_gate=True, rename=_ATTENTION)

    def _mixer_spec(self, layer: LofuvikLayer):
        m = layer.mixer
        if layer.type == "wkv":
            return WKVSpec(self.width, m["heads"], m["dim"], self.eps, rank=m.get("rank"))
        if layer.type == "delta":
            return DeltaRuleSpec(self.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], self.eps)
        right = m["right"]
        return SideBySideSpec(
            self.width, left=self._attention_spec(m["left"]),
            right=MatrixMemorySpec(self.width, right["heads"], right["dim"], right["vdim"], float(right["gate_cap"]), self.eps),
            norm_eps=self.eps)

    def _ffn_spec(self, mlp: dict) -> RoutedMLPSpec:
        # a softmax over all logits, divided by the sum of the chosen, is the softmax over the chosen
        return RoutedMLPSpec(
            hidden_size=self.width, experts=mlp["router"]["experts"], top=mlp["router"]["top"],
            expert=GatedMLPSpec(self.width, mlp["expert"]["ff"], "silu", rename=_UNIT), shared=None, score="softmax",
            renormalise=True, weight_on="output", router_bias=True)

    def runs(self) -> list:
        """(layer, pass of the loop or None) for every layer run, in order."""
        count = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(count)]
        out = [(i, None) for i in range(self.loop.start)]
        for t in range(self.loop.times):
            out += [(i, t) for i in range(self.loop.start, self.loop.stop)]
        return out + [(i, None) for i in range(self.loop.stop, count)]

    def to_model_spec(self) -> ModelSpec:
        layers = []
        for index, layer in enumerate(self.layers):
            prefix = f"l{index}"
            layers.append(LayerSpec(
                input_norm=self._norm(), mixer=self._mixer_spec(layer), post_norm=None,
                ffn=None if layer.mlp is None else self._ffn_spec(layer.mlp),
                names={"input_norm": f"{prefix}.norm1", "mixer": f"{prefix}.mix", "ffn": f"{prefix}.mlp"},
                arrangement="parallel",
            ))
        schedule = []
        for index, t in self.runs():
            schedule.append(RunSpec(index, add_embedding=bool(t) and index == self.loop.start))
        return ModelSpec(
            vocab_size=self.vocab, hidden_size=self.width, layers=tuple(layers), schedule=tuple(schedule),
            final_norm=self._norm(), tie_embeddings=False, max_positions=MAX_POSITIONS, eos_token_ids=(),
            embed_name="embed", final_norm_name="final.norm", head_name="head",
        )
