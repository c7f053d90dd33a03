"""The Lofuvik configuration reader, the checkpoint's tensor list, the scaled rotation
frequencies, the order of layer runs and the states a run keeps (no GPU)."""

from __future__ import annotations

import copy

import pytest
import torch

import plain_lofuvik as pl
from forge_engine_b200.cache.manager import CacheManager, CacheNeeds, PagedKVSpec, StateSpec
from forge_engine_b200.config import read_model_config
from forge_engine_b200.config.specs import RotarySpec
from forge_engine_b200.errors import ConfigError
from forge_engine_b200.parts.base import BuildContext, build_part, part_class


def example():
    return pl.config([
        pl.wkv_layer(),
        pl.parallel_layer(mlp=pl.routed(experts=9, top=4, ff=12)),
        pl.delta_layer(mlp=None),
        pl.parallel_layer(pl.attention_side(softcap=None, scaling=None), mlp=None),
    ], loop=(1, 3, 3))


def test_registry_finds_the_architecture_and_reads_every_constant():
    arch, _, spec = read_model_config(example())
    assert arch.name == "Lofuvik" and spec.vocab_size == 89 and spec.hidden_size == 64 and not spec.tie_embeddings
    assert all(layer.arrangement == "parallel" and layer.post_norm is None and layer.input_norm.eps == 2e-5 for layer in spec.layers)
    wkv, side, delta, plain = (layer.mixer for layer in spec.layers)
    assert wkv.kind == "wkv" and (wkv.num_heads, wkv.head_dim, wkv.rank, wkv.norm_eps) == (3, 16, None, 2e-5)
    left, right = side.left, side.right
    assert (left.num_heads, left.num_kv_heads, left.head_dim, left.v_head_dim) == (4, 2, 16, 16)
    assert left.qk_norm and left.qk_norm_scope == "whole" and left.sink and left.output_gate and not left.bias and left.window is None
    assert left.softcap == 9.0 and left.scale == pytest.approx(1.3 / 4)
    assert left.position.rotary_dim == 12 and left.position.theta == 500.0 and left.position.yarn == (4.0, 40.0, 6.0, 1.0)
    assert not left.position.interleaved and left.position.scaling is None
    assert right.kind == "matrix_memory" and (right.num_heads, right.head_dim, right.v_head_dim, right.gate_cap) == (3, 12, 20, 7.0)
    assert delta.kind == "delta_rule" and (delta.num_heads, delta.num_kv_heads, delta.head_dim, delta.v_head_dim, delta.taps) == (4, 2, 12, 20, 3)
    assert plain.left.softcap is None and plain.left.position.yarn is None
    routed = spec.layers[1].ffn
    assert (routed.experts, routed.top, routed.expert.intermediate_size, routed.expert.activation) == (9, 4, 12, "silu")
    assert routed.score == "softmax" and routed.renormalise and routed.router_bias and routed.weight_on == "output" and routed.shared is None
    assert spec.layers[2].ffn is None


def test_order_of_runs_and_where_the_embedding_joins():
    _, _, spec = read_model_config(example())
    assert [(run.layer, run.add_embedding) for run in spec.schedule] == pl.layer_runs(example())
    assert [run.layer for run in spec.schedule] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [run.add_embedding for run in spec.schedule] == [False, False, False, True, False, True, False, False]
    assert all(run.cache_of is None for run in spec.schedule)
    raw = example()
    del raw["loop"]
    assert [run.layer for run in read_model_config(raw)[2].schedule] == [0, 1, 2, 3]
    raw["loop"] = {"start": 0, "stop": 4, "times": 2}
    assert [run.add_embedding for run in read_model_config(raw)[2].schedule] == [False] * 4 + [True] + [False] * 3


def test_constants_that_may_be_left_out():
    raw = example()
    del raw["layers"][2]["mixer"]["kv_heads"], raw["layers"][1]["mixer"]["left"]["kv_heads"]
    _, _, spec = read_model_config(raw)
    assert spec.layers[2].mixer.num_kv_heads == 4 and spec.layers[1].mixer.left.num_kv_heads == 4
    del raw["layers"][1]["mixer"]["left"]["rot"]
    assert read_model_config(raw)[2].layers[1].mixer.left.position.kind == "none"


def test_expected_tensors_are_the_checkpoints():
    full = example()
    arch, _, spec = read_model_config(full)
    expected = arch.expected_tensors(spec)
    shapes = pl.tensor_shapes(full)
    assert set(expected) == set(shapes)
    for name, shape in shapes.items():
        wanted = tuple(expected[name].shape)
        assert len(wanted) == len(shape) and all(w is None or w == s for w, s in zip(wanted, shape)), name
    assert tuple(expected["l0.mix.w1"].shape) == (None, 64) and tuple(expected["l0.mix.w2"].shape) == (48, None)
    for layer in full["layers"]:
        if layer["type"] == "wkv":
            layer["mixer"]["rank"] = 5
    expected = arch.expected_tensors(read_model_config(full)[2])
    assert tuple(expected["l0.mix.w1"].shape) == (5, 64)


@pytest.mark.parametrize("path, value", (
    (("layers", 0, "type"), "attention"),
    (("layers", 0, "mixer", "heads"), 0),
    (("layers", 0, "mixer", "dim"), None),
    (("layers", 1, "mixer", "left"), None),
    (("layers", 1, "mixer", "left", "kv_heads"), 3),
    (("layers", 1, "mixer", "left", "rot", "dims"), 7),
    (("layers", 1, "mixer", "left", "rot", "dims"), 18),
    (("layers", 1, "mixer", "left", "rot", "base"), 0.0),
    (("layers", 1, "mixer", "left", "rot", "scaling", "factor"), 0.0),
    (("layers", 1, "mixer", "left", "rot", "scaling", "fast"), "x"),
    (("layers", 1, "mixer", "left", "softcap"), 0.0),
    (("layers", 1, "mixer", "left", "scale"), None),
    (("layers", 1, "mixer", "right", "gate_cap"), 0.0),
    (("layers", 1, "mixer", "right", "vdim"), -1),
    (("layers", 1, "mlp", "router", "top"), 10),
    (("layers", 1, "mlp", "kind"), "dense"),
    (("layers", 1, "mlp", "expert", "ff"), 0),
    (("layers", 2, "mixer", "conv"), 0),
    (("layers", 2, "mixer", "kv_heads"), 3),
    (("norm", "eps"), 0.0),
    (("vocab",), 0),
    (("layers",), []),
    (("loop", "stop"), 5),
    (("loop", "start"), 4),
    (("loop", "times"), 0),
))
def test_what_cannot_be_run_is_refused(path, value):
    raw = copy.deepcopy(example())
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError):
        read_model_config(raw)


@pytest.mark.parametrize("dims, base, scaling", (
    (64, 10000.0, (4.0, 2048, 32.0, 1.0)), (12, 500.0, (8.0, 40, 6.0, 1.0)), (16, 1e6, (1.0, 64, 8.0, 1.0)),
    (32, 10000.0, (16.0, 16, 1.0, 1.0)), (8, 10.0, (2.0, 100000, 2.0, 0.5)), (2, 10000.0, (4.0, 512, 32.0, 1.0)), (24, 100.0, None)))
def test_scaled_frequencies_and_amplitude(dims, base, scaling):
    rot = {"dims": dims, "base": base}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    want, amplitude = pl.frequencies(rot)
    ctx = BuildContext(dtype=torch.float32, device=torch.device("cpu"), status=None)
    part = build_part(RotarySpec(dims + 3, base, dims, exact_frequencies=True, yarn=scaling), {}, ctx)
    assert part.amplitude == pytest.approx(amplitude, rel=1e-12)
    assert torch.allclose(part.inv_freq.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-7, atol=0)


def test_the_ramp_blends_between_two_dimensions():
    """Fast turning dimensions keep their frequency, slow ones get the factor-th part."""
    from forge_engine_b200.parts.positions import RotaryEncoding

    freq = 10000.0 ** -(torch.arange(0, 64, 2, dtype=torch.float64) / 64)
    got, amplitude = RotaryEncoding.ramp(freq, 10000.0, 64, (8.0, 2048.0, 32.0, 1.0))
    ratio = got / freq
    assert float(ratio[0]) == 1.0 and float(ratio[-1]) == pytest.approx(1 / 8) and bool((ratio[1:] <= ratio[:-1]).all())
    assert amplitude == pytest.approx(1.2079441541679836)


def test_states_a_run_keeps_are_zeroed_for_a_new_request():
    needs = [CacheNeeds(kv=PagedKVSpec(2, 8), state=StateSpec((2, 3)), states=(("top", StateSpec((2,))), ("last", StateSpec((5,))))),
             CacheNeeds(state=StateSpec((4,)), states=(("top", StateSpec((7,))),)), CacheNeeds(kv=PagedKVSpec(2, 8))]
    cache = CacheManager(needs, page_size=4, num_pages=6, max_requests=2, dtype=torch.float32, device="cpu")
    view = cache.view(0)
    assert set(view.states) == {"top", "last"} and view.states["last"].shape == (3, 5) and view.state.shape == (3, 2, 3)
    assert cache.view(1).states["top"].shape == (3, 7) and cache.view(2).states == {}
    for state in (view.state, *view.states.values(), *cache.view(1).states.values()):
        state.fill_(9.0)
    entry = cache.begin_request("a")
    for state in (view.state, *view.states.values(), *cache.view(1).states.values()):
        assert float(state[entry.slot].abs().max()) == 0.0 and float(state[cache.null_slot].abs().max()) == 9.0


def test_two_mixers_side_by_side_may_not_want_the_same_place():
    _, _, spec = read_model_config(example())
    side = spec.layers[1].mixer
    shapes = part_class(side).weight_shapes(side)
    assert "left.out" in shapes and "right.i.b" in shapes and "left.q.norm" in shapes
    import dataclasses

    twice = dataclasses.replace(side, left=side.right)
    ctx = BuildContext(dtype=torch.float32, device=torch.device("cpu"), status=None)
    weights = {name: torch.zeros([e or 3 for e in info.shape]) for name, info in part_class(twice).weight_shapes(twice).items()}
    with pytest.raises(ConfigError):
        build_part(twice, weights, ctx)
