"""The Lozezen configuration reader, the checkpoint's tensor list, divided rotation frequencies and the
pages that chunks and windows give back (no GPU)."""

from __future__ import annotations

import copy

import pytest
import torch

import plain_lozezen as pl
from forge_engine_b200.cache.manager import CacheManager, CacheNeeds, PagedKVSpec
from forge_engine_b200.config import read_model_config
from forge_engine_b200.config.specs import RotarySpec
from forge_engine_b200.errors import ConfigError
from forge_engine_b200.parts.base import BuildContext, build_part


def example():
    return pl.config([
        pl.rglru_layer(width=60, blocks=4, conv=5, mlp=None),
        pl.attention_layer(heads=6, kv_heads=3, size=33, mlp=pl.dense(40)),
        pl.parallel_layer(left_scale=0.25, right_scale=-1.5, mlp=None),
        pl.attention_layer(factor=None, kv_heads=None),
        pl.rglru_layer(),
    ], eps=3e-5, scale=7.5)


def test_registry_finds_the_architecture_and_reads_every_constant():
    arch, _, spec = read_model_config(example())
    assert arch.name == "Lozezen" and (spec.vocab_size, spec.hidden_size, spec.embedding_scale) == (89, 64, 7.5) and not spec.tie_embeddings
    assert [run.layer for run in spec.schedule] == [0, 1, 2, 3, 4]
    for layer in spec.layers:
        assert layer.arrangement == "sandwich" and (layer.post_norm is None) == (layer.ffn is None) == (layer.options.ffn_out_norm is None)
        for norm in (layer.input_norm, layer.options.mixer_out_norm):
            assert (norm.eps, norm.weight_offset, norm.size) == (3e-5, 1.0, 64)
    unit, window, side, plain, _ = (layer.mixer for layer in spec.layers)
    assert unit.kind == "rglru" and (unit.width, unit.blocks, unit.taps, unit.strength) == (60, 4, 5, 8.0)
    assert window.kind == "gqa_attention" and (window.num_heads, window.num_kv_heads, window.head_dim, window.v_head_dim) == (6, 3, 16, 24)
    assert window.window == 33 and window.chunk is None and window.bias and window.o_bias is False and not window.qk_norm and not window.head_gate
    assert window.position.interleaved and (window.position.rotary_dim, window.position.theta, window.position.frequency_divisor) == (12, 300.0, 4.0)
    assert plain.position.frequency_divisor == 1.0 and plain.num_kv_heads == 4
    left, right = side.left, side.right
    assert side.scales == (0.25, -1.5)
    assert left.chunk == 18 and left.window is None and left.bias and left.head_gate and left.qk_norm and left.qk_norm_scope == "head"
    assert left.position.kind == "none" and left.scale == pytest.approx(1.4 / 12**0.5) and left.qk_norm_eps == 3e-5
    assert right.kind == "retention" and (right.num_heads, right.head_dim, right.v_head_dim, right.norm_eps) == (3, 12, 20, 3e-5)
    assert right.decay == (0.75, 0.875, 0.9375) and right.key_scale == pytest.approx(12**-0.5) and not right.norm_weight
    assert not right.position.interleaved and (right.position.rotary_dim, right.position.theta) == (8, 700.0)
    assert spec.layers[1].ffn.intermediate_size == 40 and spec.layers[1].ffn.activation == "silu" and spec.layers[2].ffn is None


def test_expected_tensors_are_the_checkpoints():
    arch, _, spec = read_model_config(example())
    assert {name: tuple(info.shape) for name, info in arch.expected_tensors(spec).items()} == pl.tensor_shapes(example())


@pytest.mark.parametrize("path, value", (
    (("layers", 0, "type"), "wkv"),
    (("layers", 0, "mixer"), None),
    (("layers", 0, "mixer", "blocks"), 7),
    (("layers", 0, "mixer", "blocks"), 0),
    (("layers", 0, "mixer", "conv"), 0),
    (("layers", 0, "mixer", "width"), 0),
    (("layers", 1, "mixer", "kv_heads"), 4),
    (("layers", 1, "mixer", "mask"), None),
    (("layers", 1, "mixer", "mask", "size"), 0),
    (("layers", 1, "mixer", "rot"), None),
    (("layers", 1, "mixer", "rot", "dims"), 5),
    (("layers", 1, "mixer", "rot", "dims"), 18),
    (("layers", 1, "mixer", "rot", "base"), 0.0),
    (("layers", 1, "mixer", "rot", "scaling", "factor"), 0.0),
    (("layers", 1, "mixer", "scale"), None),
    (("layers", 1, "mlp", "kind"), "moe"),
    (("layers", 1, "mlp", "ff"), 0),
    (("layers", 2, "mixer", "left"), None),
    (("layers", 2, "mixer", "left", "mask", "size"), -3),
    (("layers", 2, "mixer", "right", "decay"), [0.5]),
    (("layers", 2, "mixer", "right", "decay"), [0.5, 0.5, 1.5]),
    (("layers", 2, "mixer", "right", "rot", "dims"), 14),
    (("layers", 2, "mixer", "left_scale"), None),
    (("embedding", "scale"), "x"),
    (("norm", "eps"), 0.0),
    (("vocab",), 0),
    (("layers",), []),
))
def test_what_cannot_be_run_is_refused(path, value):
    raw = copy.deepcopy(example())
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError):
        read_model_config(raw)


@pytest.mark.parametrize("interleaved", (False, True))
@pytest.mark.parametrize("dims, base, factor", ((12, 300.0, 4.0), (64, 1e6, 1.0), (2, 10000.0, 3.0), (36, 30000.0, 0.5)))
def test_frequencies_are_divided_by_the_factor(dims, base, factor, interleaved):
    want = pl.angles(2, {"dims": dims, "base": base, "scaling": {"factor": factor}}, torch.float64)[1]
    ctx = BuildContext(dtype=torch.float32, device=torch.device("cpu"), status=None)
    part = build_part(RotarySpec(dims + 3, base, dims, interleaved=interleaved, exact_frequencies=True, frequency_divisor=factor), {}, ctx)
    assert torch.allclose(part.inv_freq.double(), want, rtol=1e-7, atol=0)


@pytest.mark.parametrize("size", (1, 3, 4, 8, 10, 17))
@pytest.mark.parametrize("step", (1, 2, 7))
def test_pages_of_past_chunks_are_given_back(size, step):
    """At every length exactly the pages that hold a position of the next token's chunk or a later
    one stay leased, and no more than the worst case announced."""
    spec = PagedKVSpec(2, 8, chunk=size)
    cache = CacheManager([CacheNeeds(kv=spec)], page_size=4, num_pages=40, max_requests=1)
    cache.begin_request("a")
    worst = cache.worst_case_pages(60, step)[0]
    length = 0
    while length + step <= 60:
        length += step
        cache.reserve("a", length)
        table = cache.request("a").tables[0]
        assert sum(p >= 0 for p in table.pages) <= worst
        cache.advance("a", length)
        first = length // size * size
        for index, page in enumerate(table.pages):
            assert (page >= 0) == ((index + 1) * 4 > first), (length, index)
        cache.check_consistency()
    cache.end_request("a")
    assert cache.leased_pages() == [0]


def test_what_a_cache_kind_says_of_its_reach():
    assert PagedKVSpec(1, 8).reach is None and PagedKVSpec(1, 8, 5).reach == 5 and PagedKVSpec(1, 8, chunk=6).reach == 6
    assert [PagedKVSpec(1, 8).first_needed(p) for p in (0, 9)] == [0, 0]
    assert [PagedKVSpec(1, 8, 5).first_needed(p) for p in (0, 4, 5, 9)] == [0, 0, 1, 5]
    assert [PagedKVSpec(1, 8, chunk=6).first_needed(p) for p in (0, 5, 6, 11, 12)] == [0, 0, 6, 6, 12]
    assert PagedKVSpec(1, 8, 5) != PagedKVSpec(1, 8, chunk=5)      # groups of their own
