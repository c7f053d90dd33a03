"""The Lozezen configuration: a decoder whose layers are listed one by one, with a norm on both sides of
every sublayer.

``config.json`` names the architecture in ``architecture`` and gives ``vocab``, ``width``, ``norm.eps``,
``embedding.scale`` and ``layers``.  Per layer: ``type`` (which mixer), the mixer's sizes and constants
(``mixer``) and its feed-forward (``mlp``, or null).

A layer: x += norm1b(mixer(norm1(x))), then x += norm2b(ff(norm2(x))) if it has a feed-forward.  Every norm
is an RMS norm whose weight is stored as its distance from one; the embedding rows are multiplied by
``embedding.scale``.

Mixers:

* ``rglru`` - Griffin's recurrent block around a real-gated linear recurrent unit: ``width`` channels in
  ``blocks`` parts, a convolution of ``conv`` taps;
* ``attention`` - grouped-query softmax attention with biases on q, k and v, the first ``rot.dims`` elements
  of every head rotated in neighbouring pairs (frequencies divided by ``rot.scaling.factor``), a sliding
  window of ``mask.size`` keys;
* ``parallel`` - ``left_scale`` times ``left`` plus ``right_scale`` times ``right``, both on the same input:
  ``left``, grouped-query attention with biases, q and k normalised head by head, no rotation, keys of the
  query's own chunk of ``mask.size`` positions, a sigmoid gate per head; ``right``, retention: linear
  attention with the fixed decays ``decay`` per head, q and k rotated in halves, keys times dim^(-1/2).

Feed-forward (``mlp.kind`` ``dense``): down(silu(gate(x)) * up(x)) with ``ff`` features.

Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.mix.*``, ``l<i>.norm2``, ``l<i>.norm2b``,
``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from dataclasses import dataclass

from ..errors import ConfigError
from .specs import (
    AttentionSpec,
    GatedMLPSpec,
    LayerSpec,
    ModelSpec,
    NoPositionSpec,
    NormSpec,
    RetentionSpec,
    RGLRUSpec,
    RotarySpec,
    RunSpec,
    SandwichSpec,
    SideBySideSpec,
)
from .zofadra import _int, _number

MAX_POSITIONS = 1 << 20          # rotary positions have no table; the cache bounds a request first
NORM_WEIGHT_OFFSET = 1.0         # norm weights are stored around zero
DECAY_STRENGTH = 8.0             # log a = -8 r softplus(lam)

_BARE = (("weight", ""),)        # a norm's weight is stored under the norm's own name
_ATTENTION = (("q_proj.weight", "q"), ("k_proj.weight", "k"), ("v_proj.weight", "v"), ("o_proj.weight", "o"),
              ("q_proj.bias", "q.b"), ("k_proj.bias", "k.b"), ("v_proj.bias", "v.b"),
              ("gate_proj.weight", "g"), ("q_norm.weight", "q.norm"), ("k_norm.weight", "k.norm"))
_UNIT = (("gate_proj.weight", "gate"), ("up_proj.weight", "up"), ("down_proj.weight", "down"))


@dataclass(frozen=True)
class LozezenLayer:
    type: str
    mixer: dict
    mlp: dict | None


def _check_heads(side: dict, where: str) -> dict:
    for key in ("heads", "dim", "vdim"):
        _int(side, key, where)
    if side.get("kv_heads") is None:
        side = dict(side, kv_heads=side["heads"])        # every query head with keys and values of its own
    if side["heads"] % _int(side, "kv_heads", where):
        raise ConfigError(f"{where}.heads must be a multiple of kv_heads")
    _number(side, "scale", where)
    _int(side.get("mask") or {}, "size", f"{where}.mask")
    return side


def _check_rotation(side: dict, where: str) -> None:
    rot = side.get("rot")
    if not isinstance(rot, dict):
        raise ConfigError(f"{where}.rot must be an object")
    if _number(rot, "base", f"{where}.rot") <= 0:
        raise ConfigError(f"{where}.rot.base must be positive")
    dims = _int(rot, "dims", f"{where}.rot", 2)
    if dims % 2 or dims > side["dim"]:
        raise ConfigError(f"{where}.rot.dims={dims} must be even and at most dim={side['dim']}")
    scaling = rot.get("scaling")
    if scaling is not None and _number(scaling, "factor", f"{where}.rot.scaling") <= 0:
        raise ConfigError(f"{where}.rot.scaling.factor must be positive")


def _check_mixer(kind: str, mixer: dict, where: str) -> dict:
    if kind == "rglru":
        for key in ("width", "blocks", "conv"):
            _int(mixer, key, where)
        if mixer["width"] % mixer["blocks"]:
            raise ConfigError(f"{where}.width must be a multiple of blocks")
        return mixer
    if kind == "attention":
        mixer = _check_heads(mixer, where)
        _check_rotation(mixer, where)
        return mixer
    left, right = mixer.get("left"), mixer.get("right")
    if not isinstance(left, dict) or not isinstance(right, dict):
        raise ConfigError(f"{where} must have the objects left and right")
    for key in ("heads", "dim", "vdim"):
        _int(right, key, f"{where}.right")
    _check_rotation(right, f"{where}.right")
    decay = right.get("decay")
    if not isinstance(decay, list) or len(decay) != right["heads"] or not all(
            isinstance(d, (int, float)) and not isinstance(d, bool) and 0 <= d <= 1 for d in decay):
        raise ConfigError(f"{where}.right.decay must list one number between 0 and 1 per head")
    for key in ("left_scale", "right_scale"):
        _number(mixer, key, where)
    return dict(mixer, left=_check_heads(dict(left), f"{where}.left"), right=dict(right))


@dataclass(frozen=True)
class LozezenConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: tuple

    architecture = "Lozezen"

    @classmethod
    def from_dict(cls, raw: dict) -> "LozezenConfig":
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
            if kind not in ("attention", "parallel", "rglru"):
                raise ConfigError(f"{where}.type={kind!r}; known: attention, parallel, rglru")
            mixer = _check_mixer(kind, dict(mixer), f"{where}.mixer")
            mlp = item.get("mlp")
            if mlp is not None:
                if mlp.get("kind", "dense") != "dense":
                    raise ConfigError(f"{where}.mlp.kind={mlp['kind']!r}; known: dense")
                _int(mlp, "ff", f"{where}.mlp")
            layers.append(LozezenLayer(kind, mixer, None if mlp is None else dict(mlp)))
        return cls(vocab=_int(raw, "vocab", "config"), width=_int(raw, "width", "config"), eps=eps,
                   embedding_scale=float(_number(raw.get("embedding") or {}, "scale", "embedding")), layers=tuple(layers))

    # ------------------------------------------------------------------------------
    def _norm(self) -> NormSpec:
        return NormSpec(self.width, self.eps, rename=_BARE, weight_offset=NORM_WEIGHT_OFFSET)

    @staticmethod
    def _rotary(side: dict, interleaved: bool) -> RotarySpec:
        rot = side["rot"]
        scaling = rot.get("scaling")
        return RotarySpec(head_dim=side["dim"], theta=float(rot["base"]), rotary_dim=int(rot["dims"]), interleaved=interleaved,
                          exact_frequencies=True, frequency_divisor=1.0 if scaling is None else float(scaling["factor"]))

    def _attention_spec(self, m: dict, **kind) -> AttentionSpec:
        return AttentionSpec(
            hidden_size=self.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
            qk_norm_eps=self.eps, bias=True, o_bias=False, scale=float(m["scale"]), rename=_ATTENTION, **kind)

    def _mixer_spec(self, layer: LozezenLayer):
        m = layer.mixer
        if layer.type == "rglru":
            return RGLRUSpec(self.width, m["width"], m["blocks"], m["conv"], strength=DECAY_STRENGTH)
        if layer.type == "attention":
            return self._attention_spec(m, qk_norm=False, position=self._rotary(m, interleaved=True), window=m["mask"]["size"])
        left, right = m["left"], m["right"]
        return SideBySideSpec(
            self.width,
            left=self._attention_spec(left, qk_norm=True, position=NoPositionSpec(), chunk=left["mask"]["size"], head_gate=True),
            right=RetentionSpec(self.width, right["heads"], right["dim"], right["vdim"], tuple(float(d) for d in right["decay"]), self.eps,
                                position=self._rotary(right, interleaved=False), key_scale=right["dim"] ** -0.5),
            norm_eps=self.eps, scales=(float(m["left_scale"]), float(m["right_scale"])))

    def to_model_spec(self) -> ModelSpec:
        layers = []
        for index, layer in enumerate(self.layers):
            prefix = f"l{index}"
            ffn = None if layer.mlp is None else GatedMLPSpec(self.width, layer.mlp["ff"], "silu", rename=_UNIT)
            layers.append(LayerSpec(
                input_norm=self._norm(), mixer=self._mixer_spec(layer), post_norm=None if ffn is None else self._norm(), ffn=ffn,
                names={"input_norm": f"{prefix}.norm1", "mixer": f"{prefix}.mix", "mixer_out_norm": f"{prefix}.norm1b",
                       "post_norm": f"{prefix}.norm2", "ffn": f"{prefix}.mlp", "ffn_out_norm": f"{prefix}.norm2b"},
                arrangement="sandwich",
                options=SandwichSpec(self._norm(), None if ffn is None else self._norm()),
            ))
        return ModelSpec(
            vocab_size=self.vocab, hidden_size=self.width, layers=tuple(layers),
            schedule=tuple(RunSpec(index) for index in range(len(layers))),
            final_norm=self._norm(), tie_embeddings=False, max_positions=MAX_POSITIONS, eos_token_ids=(),
            embed_name="embed", final_norm_name="final.norm", head_name="head", embedding_scale=self.embedding_scale,
        )
