"""The Lofuvik design in the engine against the plain implementation of ``plain_lofuvik.py``:
every mechanism alone, whole prompts against portions and token-by-token decoding, unequal
batches, reused pages and slots, chunk borders of the recurrences, tokens far back that reach late
logits through a state or through one loud key, sinks, the first tokens of a sequence, loops,
other sizes, generation."""

from __future__ import annotations

import json

import pytest
import torch
from safetensors.torch import save_file

import plain_lofuvik as pl

pytestmark = pytest.mark.gpu

DTYPES = ("float32", "bfloat16")


# -- helpers --------------------------------------------------------------------------------
def write_model(folder, cfg: dict, seed: int, change=None) -> dict:
    weights = pl.random_weights(cfg, seed)
    if change is not None:
        change(weights)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in weights.items()}, str(folder / "model.safetensors"))
    return weights


def make_runner(folder, dtype: str, page_size=4, num_pages=96, max_requests=4, use_graphs=True):
    from forge_engine_b200.engine import ModelRunner

    return ModelRunner.from_folder(folder, dtype=dtype, page_size=page_size, num_pages=num_pages,
                                   max_requests=max_requests, use_graphs=use_graphs)


def tokens_of(cfg: dict, length: int, seed: int, avoid=()) -> list:
    gen = torch.Generator().manual_seed(seed)
    spare = [t for t in range(cfg["vocab"]) if t not in avoid]
    return [spare[t] for t in torch.randint(0, len(spare), (length,), generator=gen).tolist()]


def run_schedule(runner, requests: dict, schedule: list) -> dict:
    """``schedule``: steps, each a list of (request, number of its next tokens); a request
    begins at its first entry and ends with its last token.  Logits of every position."""
    from forge_engine_b200.engine import StepEntry

    at = {key: 0 for key in requests}
    rows = {key: [] for key in requests}
    for step in schedule:
        entries = []
        for key, count in step:
            if at[key] == 0:
                runner.begin(key)
            entries.append(StepEntry(key, requests[key][at[key] : at[key] + count], list(range(count))))
        logits = runner.step(entries).float().cpu()
        runner.check_status()
        begin = 0
        for key, count in step:
            rows[key].append(logits[begin : begin + count])
            begin += count
            at[key] += count
            if at[key] == len(requests[key]):
                runner.end(key)
        runner.cache.check_consistency()
    assert all(at[key] == len(requests[key]) for key in requests)
    return {key: torch.cat(parts) for key, parts in rows.items()}


def assert_close(got: torch.Tensor, want: torch.Tensor, dtype: str, what: str = "") -> None:
    want = want.float()
    assert got.shape == want.shape, what
    assert torch.isfinite(got).all(), what
    scale = float(want.abs().max())
    if dtype == "float32":
        worst = float((got - want).abs().max())
        assert worst <= 2e-4 * max(1.0, scale), f"{what}: {worst} against a scale of {scale}"
    else:
        error = float(((got - want) ** 2).mean().sqrt() / (want**2).mean().sqrt())
        assert error <= 3e-2, f"{what}: relative error {error}"


def oracle(cfg, weights, tokens) -> torch.Tensor:
    return pl.forward(cfg, weights, tokens)


def routed_for(dtype: str, **kwargs):
    """A router that chooses in 32-bit; in bfloat16 one that takes every expert, because a close
    call decided the other way by rounding changes a token's logits far beyond rounding."""
    return pl.routed(**kwargs) if dtype == "float32" else pl.routed(experts=3, top=3, ff=32)


def mixed_config(dtype: str = "float32", loop=(1, 3, 2)):
    """All mechanisms in one model, the layers' head counts and sizes all different, a loop over
    the middle."""
    return pl.config([
        pl.wkv_layer(heads=3, dim=16, mlp=routed_for(dtype)),
        pl.parallel_layer(mlp=routed_for(dtype, experts=9, top=4)),
        pl.delta_layer(heads=6, kv_heads=2, dim=12, vdim=20, conv=4, mlp=None),
        pl.wkv_layer(heads=2, dim=24, mlp=None),
        pl.delta_layer(heads=2, kv_heads=2, dim=16, vdim=8, conv=2, mlp=routed_for(dtype, experts=5, top=1)),
    ], loop=loop)


# -- every mechanism alone --------------------------------------------------------------------
SINGLE = {
    "wkv": [pl.wkv_layer(mlp=None)],
    "wkv_routed": [pl.wkv_layer()],
    "wkv_one_head": [pl.wkv_layer(heads=1, dim=40, mlp=None)],
    "wkv_odd": [pl.wkv_layer(heads=5, dim=7, mlp=None)],
    "wkv_heads_of_64": [pl.wkv_layer(heads=2, dim=64, mlp=None)],
    "delta": [pl.delta_layer(mlp=None)],
    "delta_routed": [pl.delta_layer()],
    "delta_no_sharing": [pl.delta_layer(heads=3, kv_heads=3, mlp=None)],
    "delta_one_shared": [pl.delta_layer(heads=4, kv_heads=1, dim=8, vdim=8, conv=4, mlp=None)],
    "delta_one_tap": [pl.delta_layer(conv=1, mlp=None)],
    "delta_nine_taps": [pl.delta_layer(conv=9, mlp=None)],
    "delta_odd": [pl.delta_layer(heads=2, kv_heads=1, dim=9, vdim=5, mlp=None)],
    "delta_wide_values": [pl.delta_layer(heads=2, kv_heads=2, dim=32, vdim=96, mlp=None)],
    "parallel": [pl.parallel_layer(mlp=None)],
    "parallel_routed": [pl.parallel_layer()],
    "parallel_no_cap": [pl.parallel_layer(pl.attention_side(softcap=None), mlp=None)],
    "parallel_plain_frequencies": [pl.parallel_layer(pl.attention_side(scaling=None, rot_dims=16), mlp=None)],
    "parallel_two_rotated": [pl.parallel_layer(pl.attention_side(rot_dims=2), mlp=None)],
    "parallel_values_differ": [pl.parallel_layer(pl.attention_side(heads=3, kv_heads=1, dim=10, vdim=26, rot_dims=6),
                                                 pl.memory_side(heads=1, dim=9, vdim=33), mlp=None)],
    "parallel_heads_of_64": [pl.parallel_layer(pl.attention_side(heads=4, kv_heads=2, dim=64, vdim=64, rot_dims=64),
                                               pl.memory_side(heads=2, dim=48, vdim=64), mlp=None)],
    "parallel_heads_of_128": [pl.parallel_layer(pl.attention_side(heads=2, kv_heads=1, dim=128, vdim=128, rot_dims=32),
                                                pl.memory_side(heads=2, dim=32, vdim=128), mlp=None)],
    "parallel_three_per_key_head": [pl.parallel_layer(pl.attention_side(heads=6, kv_heads=2, dim=64, vdim=64, rot_dims=32),
                                                      pl.memory_side(heads=3, dim=16, vdim=16, gate_cap=30.0), mlp=None)],
    "routed_top_one": [pl.delta_layer(mlp=pl.routed(top=1))],
    "routed_all": [pl.delta_layer(mlp=pl.routed(experts=3, top=3, ff=32))],
    "routed_odd_width_of_experts": [pl.wkv_layer(mlp=pl.routed(experts=7, top=3, ff=20))],
    "routed_many": [pl.wkv_layer(mlp=pl.routed(experts=40, top=6, ff=8))],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_each_mechanism_alone(tmp_path, name, dtype):
    """A whole prompt longer than a chunk of the recurrences, then the same cut into a short
    portion, a long one and single tokens."""
    if dtype == "bfloat16" and "routed" in name and name != "routed_all":
        pytest.skip("routers that choose are compared in 32-bit and on the part alone")
    cfg = pl.config(SINGLE[name])
    weights = write_model(tmp_path / "m", cfg, 11)
    tokens = tokens_of(cfg, 137, 5)
    runner = make_runner(tmp_path / "m", dtype)
    want = oracle(cfg, weights, tokens)
    whole = run_schedule(runner, {"a": tokens}, [[("a", 137)]])["a"]
    cut = run_schedule(runner, {"b": tokens}, [[("b", 2)], [("b", 19)], [("b", 107)]] + [[("b", 1)] for _ in range(9)])["b"]
    assert_close(whole, want, dtype, name)
    assert_close(cut, want, dtype, name + ", cut")


def test_residual_after_every_layer_run(tmp_path):
    """The residual stream after every layer run, in 32-bit, against the plain implementation; a
    looped layer counts each time."""
    from forge_engine_b200.engine import StepEntry

    cfg = mixed_config(loop=(1, 4, 3))
    weights = write_model(tmp_path / "m", cfg, 12)
    tokens = tokens_of(cfg, 33, 6)
    want = []
    pl.forward(cfg, weights, tokens, layers_out=want)
    runner = make_runner(tmp_path / "m", "float32", use_graphs=False)
    seen = []
    for block in runner.model.blocks:
        inner = block.forward

        def spy(h, pending, batch, cache, inner=inner, **more):
            update = inner(h, pending, batch, cache, **more)
            seen.append((h + update.float()).cpu())
            return update

        block.forward = spy
    runner.begin("a")
    runner.step([StepEntry("a", tokens, [len(tokens) - 1])])
    runner.check_status()
    assert len(seen) == len(want) == 11
    for index, (got, ref) in enumerate(zip(seen, want)):
        assert float((got - ref.float()).abs().max()) <= 2e-4 * max(1.0, float(ref.abs().max())), f"run {index}"


@pytest.mark.parametrize("loop", (None, (0, 2, 2), (1, 3, 3), (2, 3, 4), (0, 3, 1), (1, 1, 3), (2, 3, 2)))
def test_loops(tmp_path, loop):
    """Loops at the start, in the middle, at the end, over one layer, once, over nothing; every pass
    keeps a cache and states of its own (a schedule that cuts the prompt would show a shared one)."""
    cfg = pl.config([pl.delta_layer(mlp=None), pl.parallel_layer(), pl.wkv_layer(mlp=None)], loop=loop)
    weights = write_model(tmp_path / "m", cfg, 13)
    tokens = tokens_of(cfg, 30, 3)
    runner = make_runner(tmp_path / "m", "float32")
    want = oracle(cfg, weights, tokens)
    whole = run_schedule(runner, {"a": tokens}, [[("a", 30)]])["a"]
    cut = run_schedule(runner, {"b": tokens}, [[("b", 11)], [("b", 2)], [("b", 13)]] + [[("b", 1)] for _ in range(4)])["b"]
    assert_close(whole, want, "float32", f"loop {loop}")
    assert_close(cut, want, "float32", f"loop {loop}, cut")
    if loop is not None and loop[2] > 1 and loop[0] < loop[1]:
        plain = oracle(dict(cfg, loop={"start": loop[0], "stop": loop[1], "times": 1}), weights, tokens)
        assert float((plain - want).abs().max()) > 0.05 * float(want.abs().max())


# -- the same sequence cut in different ways ------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
def test_prefill_against_token_by_token_decoding(tmp_path, dtype):
    cfg = mixed_config(dtype)
    weights = write_model(tmp_path / "m", cfg, 13)
    tokens = tokens_of(cfg, 45, 7)
    runner = make_runner(tmp_path / "m", dtype)
    ref = oracle(cfg, weights, tokens)
    whole = run_schedule(runner, {"a": tokens}, [[("a", 45)]])["a"]
    single = run_schedule(runner, {"b": tokens}, [[("b", 1)] for _ in range(45)])["b"]
    assert_close(whole, ref, dtype, "whole prompt")
    assert_close(single, ref, dtype, "token by token")


# around the chunks of 64 tokens and the 96 from which on a portion runs in chunks
SIZES = ((7, 2, 13, 3, 2, 5, 1, 16, 2, 9), (2,) * 20, (1, 2, 1, 3, 30, 2), (95, 2, 96, 3), (97, 64, 65, 1, 2), (128, 129, 2), (63, 1, 192, 4),
         (16, 17, 15, 32, 33), (160, 2, 2, 100))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", SIZES)
def test_portions_of_several_sizes(tmp_path, sizes, dtype):
    """Portions down to two tokens (and one), cut in the middle of pages and chunks, at their
    borders and one token beside them."""
    cfg = mixed_config(dtype)
    weights = write_model(tmp_path / "m", cfg, 14)
    tokens = tokens_of(cfg, sum(sizes), 8)
    runner = make_runner(tmp_path / "m", dtype)
    got = run_schedule(runner, {"a": tokens}, [[("a", n)] for n in sizes])["a"]
    assert_close(got, oracle(cfg, weights, tokens), dtype, f"portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch_against_each_alone(tmp_path, dtype):
    cfg = mixed_config(dtype)
    weights = write_model(tmp_path / "m", cfg, 15)
    requests = {"a": tokens_of(cfg, 241, 1), "b": tokens_of(cfg, 9, 2), "c": tokens_of(cfg, 123, 3), "d": tokens_of(cfg, 3, 4)}
    schedule = [
        [("a", 17), ("b", 2)],
        [("a", 1), ("b", 1), ("c", 120)],           # a long portion beside single tokens
        [("c", 2), ("a", 220), ("d", 2), ("b", 5)],
        [("d", 1), ("a", 3), ("b", 1), ("c", 1)],
    ]
    runner = make_runner(tmp_path / "m", dtype, num_pages=128)
    together = run_schedule(runner, requests, schedule)
    for key, tokens in requests.items():
        alone = run_schedule(runner, {key: tokens}, [[(key, len(tokens))]])[key]
        assert_close(together[key], oracle(cfg, weights, tokens), dtype, f"request {key} in the batch")
        if dtype == "float32":
            assert float((together[key] - alone).abs().max()) <= 1e-4 * max(1.0, float(alone.abs().max()))


@pytest.mark.parametrize("dtype", DTYPES)
def test_two_long_portions_in_one_step(tmp_path, dtype):
    """Entries whose chunks lie side by side in the scratch, none a multiple of a chunk."""
    cfg = mixed_config(dtype)
    weights = write_model(tmp_path / "m", cfg, 35)
    requests = {"a": tokens_of(cfg, 150, 1), "b": tokens_of(cfg, 203, 2), "c": tokens_of(cfg, 97, 3), "d": tokens_of(cfg, 5, 4)}
    runner = make_runner(tmp_path / "m", dtype, num_pages=160)
    got = run_schedule(runner, requests, [[("d", 3), ("a", 99), ("b", 131), ("c", 96)], [("b", 72), ("d", 2), ("c", 1), ("a", 51)]])
    for key, tokens in requests.items():
        assert_close(got[key], oracle(cfg, weights, tokens), dtype, f"request {key}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_slots_freed_and_used_again(tmp_path, dtype):
    """Two slots and a small pool: later requests get the pages and the states of earlier ones,
    which must read as new (every state: matrices, normalisers, maxima, last rows and inputs)."""
    cfg = mixed_config(dtype)
    weights = write_model(tmp_path / "m", cfg, 16)
    requests = {key: tokens_of(cfg, n, i) for i, (key, n) in enumerate((("a", 22), ("b", 31), ("c", 27), ("d", 9)))}
    schedule = [
        [("a", 20), ("b", 3)],
        [("a", 2), ("b", 20)],          # a ends
        [("c", 11), ("b", 1)],          # c takes a's slot and pages
        [("b", 7), ("c", 16)],          # both end
        [("d", 9)],
    ]
    runner = make_runner(tmp_path / "m", dtype, page_size=4, num_pages=16, max_requests=2)
    got = run_schedule(runner, requests, schedule)
    assert runner.cache.slots.leased_count == 0 and all(n == 0 for n in runner.cache.leased_pages())
    for key, tokens in requests.items():
        assert_close(got[key], oracle(cfg, weights, tokens), dtype, f"request {key}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(tmp_path, dtype):
    """A short prompt, then more single tokens than a chunk holds; the steps are replayed from
    captured graphs."""
    cfg = mixed_config(dtype)
    weights = write_model(tmp_path / "m", cfg, 17)
    tokens = tokens_of(cfg, 150, 9)
    runner = make_runner(tmp_path / "m", dtype, page_size=4, num_pages=40)
    got = run_schedule(runner, {"a": tokens}, [[("a", 5)]] + [[("a", 1)] for _ in range(145)])["a"]
    assert_close(got, oracle(cfg, weights, tokens), dtype, "long decoding")
    assert runner.use_graphs and runner.graphs.captured


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", (16, 100))
def test_mixed_steps_replayed_from_graphs(tmp_path, portion, dtype):
    """Steps that bring a prompt portion beside two decoding requests, captured at first sight
    and replayed (filler entries pad them to their bucket), with portions that are walked and
    portions that run in chunks.  Logits at every entry's last token."""
    from forge_engine_b200.engine import StepEntry

    cfg = mixed_config(dtype)
    weights = write_model(tmp_path / "m", cfg, 18)
    requests = {"a": tokens_of(cfg, portion * 4 + 5, 1), "b": tokens_of(cfg, 14, 2), "c": tokens_of(cfg, 19, 3)}
    schedule = [[("b", 9), ("c", 14)]] + [[("a", portion), ("b", 1), ("c", 1)] for _ in range(4)] + [[("a", 5), ("b", 1), ("c", 1)]]
    runner = make_runner(tmp_path / "m", dtype, page_size=16, num_pages=40)
    runner.graphs.capture_after = 1
    refs = {key: oracle(cfg, weights, tokens).float() for key, tokens in requests.items()}
    at = {key: 0 for key in requests}
    for step in schedule:
        entries = []
        for key, count in step:
            if at[key] == 0:
                runner.begin(key)
            entries.append(StepEntry(key, requests[key][at[key] : at[key] + count], [count - 1]))
        logits = runner.step(entries).float().cpu()
        runner.check_status()
        for row, (key, count) in enumerate(step):
            at[key] += count
            assert_close(logits[row : row + 1], refs[key][at[key] - 1 : at[key]], dtype, f"{key} at {at[key] - 1}")
    assert len(runner.graphs.captured) >= 1


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_first_tokens_of_a_sequence(tmp_path, dtype):
    """Sequences of one to five tokens, alone and side by side, in slots and pages that hold an
    earlier request's keys and states: no row before the first, no earlier inputs of the
    convolution, a maximum of zero."""
    cfg = mixed_config(dtype)
    weights = write_model(tmp_path / "m", cfg, 25)
    runner = make_runner(tmp_path / "m", dtype, max_requests=4, num_pages=24)
    warm = {key: tokens_of(cfg, 12, 40 + i) for i, key in enumerate("wxyz")}
    run_schedule(runner, warm, [[(key, 12) for key in warm]])
    requests = {key: tokens_of(cfg, n, 30 + n) for key, n in (("a", 1), ("b", 2), ("c", 3), ("d", 5))}
    got = run_schedule(runner, requests, [[("a", 1), ("b", 1), ("c", 3), ("d", 2)], [("b", 1), ("d", 3)]])
    for key, tokens in requests.items():
        assert_close(got[key], oracle(cfg, weights, tokens), dtype, f"request {key}")


# -- other sizes ------------------------------------------------------------------------------
OTHER = {
    "narrow": dict(layers=[pl.wkv_layer(heads=1, dim=4, mlp=None), pl.delta_layer(heads=1, kv_heads=1, dim=4, vdim=4, conv=2, mlp=None),
                           pl.parallel_layer(pl.attention_side(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2),
                                             pl.memory_side(heads=1, dim=4, vdim=4), mlp=pl.routed(experts=1, top=1, ff=8))], width=20, vocab=11),
    "width_not_in_eights": dict(layers=[pl.wkv_layer(heads=2, dim=10), pl.delta_layer(mlp=None), pl.parallel_layer()], width=36),
    "every_head_its_own_keys": dict(layers=[pl.parallel_layer(pl.attention_side(heads=4, kv_heads=4), mlp=None),
                                            pl.delta_layer(heads=4, kv_heads=4, mlp=None)]),
    "many_heads_per_key_head": dict(layers=[pl.parallel_layer(pl.attention_side(heads=12, kv_heads=1, dim=8, vdim=8, rot_dims=4), mlp=None),
                                            pl.delta_layer(heads=12, kv_heads=1, dim=8, vdim=8, mlp=None)]),
    "many_state_heads": dict(layers=[pl.wkv_layer(heads=16, dim=8, mlp=None),
                                     pl.parallel_layer(right=pl.memory_side(heads=16, dim=8, vdim=8), mlp=None)]),
    "wide_heads": dict(layers=[pl.wkv_layer(heads=1, dim=128, mlp=None), pl.delta_layer(heads=1, kv_heads=1, dim=128, vdim=128, mlp=None),
                               pl.parallel_layer(right=pl.memory_side(heads=1, dim=128, vdim=128), mlp=None)], width=96),
    "wider_heads": dict(layers=[pl.wkv_layer(heads=1, dim=192, mlp=None), pl.delta_layer(heads=1, kv_heads=1, dim=200, vdim=256, mlp=None),
                                pl.parallel_layer(right=pl.memory_side(heads=1, dim=160, vdim=250), mlp=None)], width=96),
    "scale_one_eps_large": dict(layers=[pl.parallel_layer(pl.attention_side(scale=1.0)), pl.wkv_layer(), pl.delta_layer()], eps=0.5),
    "caps_of_one": dict(layers=[pl.parallel_layer(pl.attention_side(softcap=1.0), pl.memory_side(gate_cap=1.0))]),
    "factor_of_one": dict(layers=[pl.parallel_layer(pl.attention_side(scaling=(1.0, 64, 8.0, 1.0)), mlp=None)]),
    "equal_ramp_ends": dict(layers=[pl.parallel_layer(pl.attention_side(scaling=(8.0, 16, 1.0, 1.0)), mlp=None)]),
    "long_original": dict(layers=[pl.parallel_layer(pl.attention_side(scaling=(16.0, 4096, 32.0, 1.0), base=10000.0, rot_dims=16), mlp=None)]),
    "top_equals_experts": dict(layers=[pl.delta_layer(mlp=pl.routed(experts=4, top=4))]),
    "one_kind_only": dict(layers=[pl.delta_layer(mlp=pl.routed(top=1)), pl.delta_layer(), pl.delta_layer(mlp=None)], loop=(0, 3, 2)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(OTHER))
def test_other_sizes_and_values_that_are_one_or_equal(tmp_path, name, dtype):
    options = dict(OTHER[name])
    layers = options.pop("layers")
    if dtype == "bfloat16":      # no router that chooses
        layers = [dict(layer, mlp=layer["mlp"] and pl.routed(experts=2, top=2, ff=layer["mlp"]["expert"]["ff"])) for layer in layers]
    cfg = pl.config(layers, **options)
    weights = write_model(tmp_path / "m", cfg, 21)
    tokens = tokens_of(cfg, 140, 10)
    runner = make_runner(tmp_path / "m", dtype, page_size=8, num_pages=48)
    ref = oracle(cfg, weights, tokens)
    whole = run_schedule(runner, {"a": tokens}, [[("a", 140)]])["a"]
    cut = run_schedule(runner, {"b": tokens}, [[("b", 19)], [("b", 2)], [("b", 101)], [("b", 2)]] + [[("b", 1)] for _ in range(16)])["b"]
    assert_close(whole, ref, dtype, name)
    assert_close(cut, ref, dtype, name + ", cut")


@pytest.mark.parametrize("rank", (1, 3, 48))
def test_ranks_of_the_decay(tmp_path, rank):
    """No key of the configuration gives the rank of the decay's two matrices: the tensors do."""
    cfg = pl.config([pl.wkv_layer(mlp=None)])
    weights = pl.random_weights(cfg, 4, rank=rank)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(weights, str(tmp_path / "model.safetensors"))
    tokens = tokens_of(cfg, 30, 1)
    got = run_schedule(make_runner(tmp_path, "float32"), {"a": tokens}, [[("a", 22)], [("a", 7)], [("a", 1)]])["a"]
    assert_close(got, oracle(cfg, weights, tokens), "float32", f"rank {rank}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_of_the_tensor_core_paths(tmp_path, dtype):
    """Sizes in sixteens, so that the bfloat16 engine takes its tensor-core products and both
    tensor-core attention kernels, with steps long enough for several row tiles and key tiles."""
    all_of_them = pl.routed(experts=3, top=3, ff=64)
    cfg = pl.config([pl.wkv_layer(heads=2, dim=64, mlp=all_of_them),
                     pl.parallel_layer(pl.attention_side(heads=4, kv_heads=2, dim=64, vdim=64, rot_dims=64, scaling=(4.0, 256, 16.0, 1.0)),
                                       pl.memory_side(heads=2, dim=32, vdim=64), mlp=all_of_them),
                     pl.delta_layer(heads=4, kv_heads=2, dim=32, vdim=64, mlp=None),
                     pl.parallel_layer(pl.attention_side(heads=2, kv_heads=1, dim=128, vdim=128, rot_dims=96, scale=0.1, softcap=20.0),
                                       pl.memory_side(heads=2, dim=64, vdim=64), mlp=None)], width=128)
    weights = write_model(tmp_path / "m", cfg, 22)
    tokens = tokens_of(cfg, 400, 11)
    runner = make_runner(tmp_path / "m", dtype, page_size=16, num_pages=64)
    ref = oracle(cfg, weights, tokens)
    whole = run_schedule(runner, {"a": tokens}, [[("a", 400)]])["a"]
    cut = run_schedule(runner, {"b": tokens}, [[("b", 130)], [("b", 2)], [("b", 200)], [("b", 63)]] + [[("b", 1)] for _ in range(5)])["b"]
    assert_close(whole, ref, dtype, "whole")
    assert_close(cut, ref, dtype, "cut")


# -- far tokens --------------------------------------------------------------------------------
def loud_pair(cfg: dict, weights: dict, key_token: int, query_token: int, wish: float) -> None:
    """Make the key of ``key_token`` point where the query of ``query_token`` points in every head
    of the first layer's attention, and set the score scale so that the pair's score is ``wish``
    in the weakest head: that key then takes nearly all of that query's weight."""
    m, p = cfg["layers"][0]["mixer"]["left"], "l0.mix.left."
    heads, kv_heads, dim, rot, eps = m["heads"], m["kv_heads"], m["dim"], m["rot"]["dims"], cfg["norm"]["eps"]
    w = {k: v.double() for k, v in weights.items()}
    row = lambda token: pl.rms(weights["embed"][token].double(), eps) * w["l0.norm1"]  # noqa: E731
    query = lambda token: (pl.rms(w[p + "q"] @ row(token), eps) * w[p + "q.norm"]).view(kv_heads, heads // kv_heads, dim)  # noqa: E731
    target = query(query_token).mean(dim=1)
    target[:, :rot] = 0.0                                    # the rotated elements turn with the distance
    h = torch.linalg.lstsq(w[p + "k"], (target.reshape(-1) / w[p + "k.norm"])[:, None]).solution[:, 0]
    embed = h / w["l0.norm1"]
    weights["embed"][key_token] = (embed / embed.pow(2).mean().sqrt()).to(weights["embed"].dtype)
    key = (pl.rms(w[p + "k"] @ row(key_token), eps) * w[p + "k.norm"]).view(kv_heads, dim)
    score = (query(query_token)[:, :, rot:] * key[:, None, rot:]).sum(-1)
    assert float(score.min()) > 0
    m["scale"] = wish / float(score.min())


FAR = {
    "plain": pl.attention_side(heads=4, kv_heads=2, dim=32, vdim=32, rot_dims=2, base=1e6, scaling=None, softcap=80.0),
    "heads_of_64": pl.attention_side(heads=2, kv_heads=1, dim=64, vdim=64, rot_dims=4, base=1e6, scaling=(4.0, 64, 8.0, 1.0), softcap=None),
    "heads_of_64_capped": pl.attention_side(heads=2, kv_heads=1, dim=64, vdim=64, rot_dims=4, base=1e6, softcap=60.0),
    "heads_of_128": pl.attention_side(heads=2, kv_heads=1, dim=128, vdim=128, rot_dims=8, base=1e6, scaling=None, softcap=70.0),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", sorted(FAR))
def test_one_loud_key_far_back_and_at_page_borders(tmp_path, kind, dtype):
    """One layer, one key that takes nearly all the weight of every loud query after it: at the
    first position, before and after page and key-tile borders, hundreds of tokens back, read by a
    prompt's own portion, by later portions and by decoded tokens."""
    cfg = pl.config([pl.parallel_layer(dict(FAR[kind]), pl.memory_side(), mlp=None)], width=192, vocab=40)
    key_token, query_token = 38, 39

    def change(weights):
        weights["l0.mix.left.sink"] = torch.full_like(weights["l0.mix.left.sink"], -1.0)
        loud_pair(cfg, weights, key_token, query_token, 22.0)

    change(pl.random_weights(cfg, 23))            # sets the scale in cfg before the folder is written
    weights = write_model(tmp_path / "m", cfg, 23, change=change)
    length = 330
    runner = make_runner(tmp_path / "m", dtype, page_size=16, num_pages=64)
    for at in (0, 15, 16, 127, 128, 200):
        tokens = tokens_of(cfg, length, 12, avoid=(key_token, query_token))
        plain = list(tokens)
        tokens[at] = key_token
        queries = [q for q in (at + 1, at + 16, 255, 256, 300, 325) if q > at]
        for q in queries:
            tokens[q] = plain[q] = query_token
        ref, without = oracle(cfg, weights, tokens), oracle(cfg, weights, plain)
        for q in queries:
            assert float(((ref[q] - without[q]) ** 2).mean().sqrt() / (ref[q] ** 2).mean().sqrt()) > 0.2, "the key decides the logits there"
        whole = run_schedule(runner, {"a": tokens}, [[("a", length)]])["a"]
        cut = run_schedule(runner, {"b": tokens}, [[("b", at + 1)], [("b", 70)], [("b", length - at - 91)]] + [[("b", 1)] for _ in range(20)])["b"]
        for got, what in ((whole, "prompt"), (cut, "cut")):
            assert_close(got, ref, dtype, f"{what}, key at {at}")
            for q in queries:
                assert_close(got[q : q + 1], ref[q : q + 1], dtype, f"{what}, key at {at}, query at {q}")


def slow_decay(weights: dict) -> None:
    """Gates and decays close to keeping everything."""
    for name, t in weights.items():
        if name.endswith(".w0"):
            weights[name] = torch.full_like(t, -7.0)
        elif name.endswith("A_log"):
            weights[name] = torch.full_like(t, -6.0)
        elif name.endswith("right.f.b"):
            weights[name] = torch.full_like(t, 6.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ("wkv", "delta", "parallel"))
def test_a_token_far_back_reaches_late_logits_through_the_state(tmp_path, kind, dtype):
    """States that hardly decay: a token changed at the start, at chunk borders or beside them moves
    the logits hundreds of tokens later, in prompts, in later portions and in decoding."""
    layer = {"wkv": pl.wkv_layer(heads=2, dim=32, mlp=None), "delta": pl.delta_layer(heads=2, kv_heads=1, dim=32, vdim=32, mlp=None),
             "parallel": pl.parallel_layer(pl.attention_side(), pl.memory_side(heads=2, dim=32, vdim=32), mlp=None)}[kind]
    cfg = pl.config([layer])
    weights = write_model(tmp_path / "m", cfg, 24, change=slow_decay)
    runner = make_runner(tmp_path / "m", dtype, page_size=16, num_pages=64)
    tokens = tokens_of(cfg, 300, 13)
    first = oracle(cfg, weights, tokens)
    for at in (0, 63, 64, 127, 130):
        ids = list(tokens)
        ids[at] = (ids[at] + 7) % cfg["vocab"]
        ref = oracle(cfg, weights, ids)
        assert float((ref[-1] - first[-1]).abs().max()) > 1e-3 * float(first[-1].abs().max())
        whole = run_schedule(runner, {"a": ids}, [[("a", 300)]])["a"]
        cut = run_schedule(runner, {"b": ids}, [[("b", 64)], [("b", 2)], [("b", 214)]] + [[("b", 1)] for _ in range(20)])["b"]
        assert_close(whole, ref, dtype, f"changed at {at}")
        assert_close(cut, ref, dtype, f"changed at {at}, cut")
        if dtype == "float32":      # the effect itself, not only the logits it is part of
            change = (ref - first)[-20:].float()
            before = run_schedule(runner, {"c": tokens}, [[("c", 300)]])["c"][-20:]
            assert float(((whole[-20:] - before) - change).abs().max()) <= 0.02 * float(change.abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", (dict(), dict(dim=64, vdim=64), dict(dim=64, vdim=64, heads=6, kv_heads=2)),
                         ids=("plain kernel", "tensor cores", "general tensor cores"))
def test_sinks_take_their_share(tmp_path, sizes, dtype):
    """Sinks from far below to far above the scores, one per head; counted once however the keys
    are split over blocks (decoding far into a long context splits them), neither scaled nor capped."""
    side = pl.attention_side(softcap=3.0, **sizes)
    cfg = pl.config([pl.parallel_layer(side, pl.memory_side(), mlp=None)])

    def change(weights):
        weights["l0.mix.left.sink"] = torch.linspace(-30.0, 9.0, side["heads"]).to(torch.bfloat16)

    weights = write_model(tmp_path / "m", cfg, 26, change=change)
    tokens = tokens_of(cfg, 280, 14)
    ref = oracle(cfg, weights, tokens)
    flat = dict(weights)
    flat["l0.mix.left.sink"] = torch.full_like(weights["l0.mix.left.sink"], -1e4)
    assert float(((ref - oracle(cfg, flat, tokens)) ** 2).mean().sqrt() / (ref**2).mean().sqrt()) > 0.05
    runner = make_runner(tmp_path / "m", dtype, page_size=16, num_pages=32)
    whole = run_schedule(runner, {"a": tokens}, [[("a", 280)]])["a"]
    decoded = run_schedule(runner, {"b": tokens}, [[("b", 250)]] + [[("b", 1)] for _ in range(30)])["b"]
    assert_close(whole, ref, dtype, "prompt")
    assert_close(decoded, ref, dtype, "decoded")


# -- parts and kernels alone -------------------------------------------------------------------
def entry_tensors(counts: list):
    cu = [0]
    for n in counts:
        cu.append(cu[-1] + n)
    entry = [e for e, n in enumerate(counts) for _ in range(n)]
    make = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")  # noqa: E731
    return make(cu), make(entry), make(list(range(len(counts)))[::-1])      # slots in reverse order of the entries


def status_word():
    return torch.zeros(1, dtype=torch.int32, device="cuda")


SHAPES = ((2, 8, 8), (3, 12, 20), (1, 64, 64), (2, 48, 64), (1, 128, 128), (1, 100, 36), (1, 256, 320), (2, 33, 7))
COUNTS = ([1, 1, 1], [5, 1, 95], [96, 3, 130], [200])


@pytest.mark.parametrize("counts", COUNTS)
@pytest.mark.parametrize("heads, dk, dv", [s for s in SHAPES])
def test_delta_rule_kernels(heads, dk, dv, counts):
    """From states that are not zero; decays from hardly any to almost total, beta near 0 and 1, keys
    that repeat (the triangular system is then far from the identity)."""
    from forge_engine_b200.ops import native

    gen = torch.Generator().manual_seed(dk * 7 + dv)
    n, kv = sum(counts), 1
    qkv = torch.randn(n, 2 * kv * dk + heads * dv, generator=gen, dtype=torch.float64)
    qkv[:, :dk], qkv[:, dk : 2 * dk] = pl.unit(qkv[:, :dk]) * dk**-0.5, pl.unit(qkv[:, dk : 2 * dk])
    qkv[1::3, dk : 2 * dk] = qkv[0, dk : 2 * dk]
    log_g = -torch.exp(4.0 * torch.randn(n, heads, generator=gen, dtype=torch.float64) - 3.0).clamp(max=60.0)
    beta = torch.sigmoid(4.0 * torch.randn(n, heads, generator=gen, dtype=torch.float64))
    gate, norm = torch.randn(n, heads * dv, generator=gen, dtype=torch.float64), 1 + 0.1 * torch.randn(dv, generator=gen, dtype=torch.float64)
    state = 0.5 * torch.randn(len(counts) + 1, heads, dk, dv, generator=gen, dtype=torch.float64)
    cu, _, slots = entry_tensors(counts)
    want, want_state = torch.empty(n, heads, dv, dtype=torch.float64), state.clone()
    for e in range(len(counts)):
        for h in range(heads):
            S = want_state[slots[e], h]
            for t in range(cu[e], cu[e + 1]):
                q, k, v = qkv[t, :dk], qkv[t, dk : 2 * dk], qkv[t, 2 * dk :].view(heads, dv)[h]
                S *= torch.exp(log_g[t, h])
                S += torch.outer(k, beta[t, h] * (v - S.T @ k))
                want[t, h] = S.T @ q
    want = (pl.rms(want, 1e-5) * norm * pl.silu(gate.view(n, heads, dv))).view(n, heads * dv)
    dev = lambda t: t.float().cuda().contiguous()  # noqa: E731
    got_state, out, status = dev(state), torch.empty(n, heads * dv, device="cuda"), status_word()
    native.delta_rule(dev(qkv), dev(torch.stack([beta, log_g], dim=-1)), dev(gate), dev(norm), 1e-5, got_state, slots, cu, out, kv,
                      len(counts), max(counts), status)
    assert int(status.item()) == 0 and not native.damaged_canaries()
    assert float((out.cpu() - want).abs().max()) <= 3e-4 * max(1.0, float(want.abs().max()))
    assert float((got_state.cpu() - want_state).abs().max()) <= 3e-5 * max(1.0, float(want_state.abs().max()))


@pytest.mark.parametrize("counts", COUNTS)
@pytest.mark.parametrize("heads, dim", ((2, 8), (3, 20), (1, 64), (1, 128), (2, 33), (1, 192), (1, 272)))
def test_wkv_kernels(heads, dim, counts):
    """Decays from 1 to 0 exactly (exp(-exp(.)) underflows), from states that are not zero."""
    from forge_engine_b200.ops import native

    gen = torch.Generator().manual_seed(dim)
    n, size = sum(counts), heads * dim
    r, k, v, gate = torch.randn(4, n, size, generator=gen, dtype=torch.float64)
    decay = torch.exp(-torch.exp(4.0 * torch.randn(n, size, generator=gen, dtype=torch.float64) - 2.0))
    u, norm = torch.randn(heads, dim, generator=gen, dtype=torch.float64), 1 + 0.1 * torch.randn(size, generator=gen, dtype=torch.float64)
    state = 0.5 * torch.randn(len(counts) + 1, heads, dim, dim, generator=gen, dtype=torch.float64)
    cu, _, slots = entry_tensors(counts)
    want, want_state = torch.empty(n, heads, dim, dtype=torch.float64), state.clone()
    at = lambda x, t, h: x[t].view(heads, dim)[h]  # noqa: E731
    for e in range(len(counts)):
        for h in range(heads):
            S = want_state[slots[e], h]
            for t in range(cu[e], cu[e + 1]):
                write = torch.outer(at(k, t, h), at(v, t, h))
                want[t, h] = (S + u[h][:, None] * write).T @ at(r, t, h)
                S.copy_(at(decay, t, h)[:, None] * S + write)
    want = pl.rms(want, 1e-5).view(n, size) * norm * pl.silu(gate)
    dev = lambda t: t.float().cuda().contiguous()  # noqa: E731
    got_state, out, status = dev(state), torch.empty(n, size, device="cuda"), status_word()
    native.wkv(dev(r), dev(k), dev(v), dev(decay), dev(u), dev(norm), dev(gate), 1e-5, got_state, slots, cu, out, len(counts), max(counts), status)
    assert int(status.item()) == 0 and not native.damaged_canaries()
    assert float((out.cpu() - want).abs().max()) <= 3e-4 * max(1.0, float(want.abs().max()))
    assert float((got_state.cpu() - want_state).abs().max()) <= 3e-5 * max(1.0, float(want_state.abs().max()))


@pytest.mark.parametrize("cap", (0.5, 9.0, 40.0))
@pytest.mark.parametrize("counts", COUNTS)
@pytest.mark.parametrize("heads, dk, dv", [s for s in SHAPES])
def test_matrix_memory_kernels(heads, dk, dv, counts, cap):
    """Gates over the whole range the cap allows (with a cap of 40 a chunk's sum of log forget gates
    falls below -1000), from states with a maximum that is not zero."""
    from forge_engine_b200.ops import native

    gen = torch.Generator().manual_seed(dk + 3 * dv)
    n = sum(counts)
    rand = lambda *shape: torch.randn(*shape, generator=gen, dtype=torch.float64)  # noqa: E731
    q, k, v, gate = rand(n, heads, dk), rand(n, heads, dk), rand(n, heads, dv), rand(n, heads, dv)
    zi, zf, bi, bf = 2 * cap * rand(n, heads), 2 * cap * rand(n, heads) + 0.5 * cap, rand(heads), rand(heads)
    log_in = cap * torch.tanh((zi + bi) / cap)
    log_forget = pl.log_sigmoid(cap * torch.tanh((zf + bf) / cap))
    state, normaliser, top = 0.5 * rand(len(counts) + 1, heads, dk, dv), 0.5 * rand(len(counts) + 1, heads, dk), rand(len(counts) + 1, heads).abs()
    norm = 1 + 0.1 * rand(heads * dv)
    cu, _, slots = entry_tensors(counts)
    want, want_state, want_n, want_top = torch.empty(n, heads, dv, dtype=torch.float64), state.clone(), normaliser.clone(), top.clone()
    for e in range(len(counts)):
        s = int(slots[e])
        for h in range(heads):
            for t in range(cu[e], cu[e + 1]):
                f, i, m = log_forget[t, h], log_in[t, h], want_top[s, h].clone()
                new = torch.maximum(f + m, i)
                want_state[s, h] = torch.exp(f + m - new) * want_state[s, h] + torch.exp(i - new) * torch.outer(k[t, h], v[t, h])
                want_n[s, h] = torch.exp(f + m - new) * want_n[s, h] + torch.exp(i - new) * k[t, h]
                want_top[s, h] = new
                qt = q[t, h] * dk**-0.5
                want[t, h] = want_state[s, h].T @ qt / (torch.maximum((want_n[s, h] @ qt).abs(), torch.exp(-new)) + 1e-6)
    raw = want
    want = pl.rms(want, 1e-5).view(n, heads * dv) * norm * pl.sigmoid(gate.view(n, -1))
    dev = lambda t: t.float().cuda().contiguous()  # noqa: E731
    proj = torch.cat([x.reshape(n, -1) for x in (q, k, v, gate, zi, zf)], dim=1)
    sizes = [heads * dk, heads * dk, heads * dv, heads * dv, heads]
    offsets = [sum(sizes[:j]) for j in range(6)]
    got = [dev(x) for x in (state, normaliser, top)]
    out, status = torch.empty(n, heads * dv, device="cuda"), status_word()
    native.matrix_memory(dev(proj), offsets, dev(bi), dev(bf), cap, dk**-0.5, dev(norm), 1e-5, *got, slots, cu, out, len(counts), max(counts), status)
    assert int(status.item()) == 0 and not native.damaged_canaries()
    # rows whose output nearly cancels are divided by a tiny root mean square: compare where it is not tiny
    clear = (raw.pow(2).mean(-1) > 1e-4).repeat_interleave(dv, dim=1).view(n, heads * dv)
    assert n < 20 or float(clear.float().mean()) > 0.5
    assert float(((out.cpu() - want).abs() * clear).max()) <= 2e-3 * max(1.0, float(want.abs().max()))
    for mine, ref, what in zip(got, (want_state, want_n, want_top), ("state", "normaliser", "maximum")):
        assert float((mine.cpu() - ref).abs().max()) <= 1e-4 * max(1.0, float(ref.abs().max())), what


@pytest.mark.parametrize("taps", (1, 2, 4, 9))
@pytest.mark.parametrize("counts", ([1, 1], [1, 5, 2], [30, 3, 8]))
def test_delta_prepare_kernel(taps, counts):
    from forge_engine_b200.ops import native

    gen = torch.Generator().manual_seed(taps)
    heads, kv, dk, dv, n = 4, 2, 6, 10, sum(counts)
    channels = 2 * kv * dk + heads * dv
    rand = lambda *shape: torch.randn(*shape, generator=gen, dtype=torch.float64)  # noqa: E731
    proj, conv, a_log, dt = rand(n, channels + heads * dv + 2 * heads), rand(channels, taps), rand(heads), rand(heads)
    state = rand(len(counts) + 1, taps - 1, channels)
    cu, entry, slots = entry_tensors(counts)
    want, want_state = torch.empty(n, channels, dtype=torch.float64), state.clone()
    for e in range(len(counts)):
        rows = torch.cat([state[slots[e]], proj[cu[e] : cu[e + 1], :channels]])
        mixed = pl.silu(sum(rows[j : j + counts[e]] * conv[:, j] for j in range(taps)))
        q, k, v = mixed.split([kv * dk, kv * dk, heads * dv], dim=1)
        unit = lambda x: pl.unit(x.reshape(-1, kv, dk)).reshape(-1, kv * dk)  # noqa: E731
        want[cu[e] : cu[e + 1]] = torch.cat([unit(q) * dk**-0.5, unit(k), v], dim=1)
        want_state[slots[e]] = rows[len(rows) - (taps - 1):]
    b, a = proj[:, -2 * heads : -heads], proj[:, -heads:]
    want_gates = torch.stack([pl.sigmoid(b), -torch.exp(a_log) * pl.softplus(a + dt)], dim=-1)
    dev = lambda t: t.float().cuda().contiguous()  # noqa: E731
    got_state = dev(state)
    out, gates = torch.empty(n, channels, device="cuda"), torch.empty(n, heads, 2, device="cuda")
    native.delta_prepare(dev(proj), channels + heads * dv, channels + heads * dv + heads, dev(conv.T), got_state if taps > 1 else None, slots,
                         cu, entry, dev(a_log), dev(dt), kv, dk, heads, dv, out, gates, len(counts))
    for mine, ref in ((out, want), (gates, want_gates), (got_state, want_state)):
        if ref.numel():
            assert float((mine.cpu() - ref).abs().max()) <= 2e-5 * max(1.0, float(ref.abs().max()))


@pytest.mark.parametrize("dtype", (torch.float32, torch.bfloat16))
@pytest.mark.parametrize("counts", ([1, 1, 1], [1, 4, 2]))
@pytest.mark.parametrize("width", (20, 1024))
def test_token_shift_kernel(width, counts, dtype):
    """From normalised rows, and - where every entry brings one token - with sum and norm in the same launch."""
    from forge_engine_b200.ops import native

    gen = torch.Generator().manual_seed(width)
    rand = lambda *shape: torch.randn(*shape, generator=gen, dtype=torch.float64)  # noqa: E731
    n = sum(counts)
    x, update, extra, weight, mu, state = rand(n, width), rand(n, width), rand(n, width), rand(width), rand(5, width), rand(len(counts) + 1, width)
    cu, entry, slots = entry_tensors(counts)
    total = x + update + extra
    h = pl.rms(total, 1e-5) * weight
    before, want_state = torch.empty_like(h), state.clone()
    for e in range(len(counts)):
        before[cu[e] : cu[e + 1]] = torch.cat([state[slots[e]][None], h[cu[e] : cu[e + 1] - 1]])
        want_state[slots[e]] = h[cu[e + 1] - 1]
    want = h + (before - h) * mu[:, None, :]
    dev = lambda t: t.float().cuda().contiguous()  # noqa: E731
    fused = {"y": dev(h)} if max(counts) > 1 else {"residual": dev(x), "update": dev(update), "shift": dev(extra), "weight": dev(weight), "eps": 1e-5}
    got_state, mixed, rows = dev(state), torch.empty(5, n, width, dtype=dtype, device="cuda"), torch.empty(n, width, dtype=dtype, device="cuda")
    native.token_shift(dev(mu), got_state, slots, cu, entry, mixed, rows, **fused)
    tol = 2e-5 if dtype == torch.float32 else 8e-3
    for mine, ref in ((mixed, want), (rows, h)):
        assert float((mine.float().cpu() - ref).abs().max()) <= tol * float(ref.abs().max())
    assert float((got_state.cpu() - want_state).abs().max()) <= 2e-5 * float(want_state.abs().max())
    if "residual" in fused:
        assert float((fused["residual"].cpu() - total).abs().max()) <= 1e-5


@pytest.mark.parametrize("dtype", (torch.float32, torch.bfloat16))
@pytest.mark.parametrize("experts, top, tokens, ff", ((6, 2, 150, 32), (12, 5, 300, 96), (5, 1, 5, 40), (30, 6, 64, 16), (9, 3, 90, 20)))
def test_routed_feed_forward_alone(experts, top, tokens, ff, dtype):
    """The part alone against a loop over tokens and experts, with a row of another sublayer that
    joins in its last kernel.  Tokens whose choice is not clear are left out."""
    from forge_engine_b200.config.specs import GatedMLPSpec, RoutedMLPSpec
    from forge_engine_b200.parts.base import BuildContext, build_part

    gen = torch.Generator().manual_seed(experts * 10 + top)
    width = 48
    mlp = pl.routed(experts=experts, top=top, ff=ff)
    cfg = pl.config([pl.delta_layer(mlp=mlp)], width=width)
    weights = {name[len("l0.mlp."):]: t for name, t in pl.random_weights(cfg, 7).items() if name.startswith("l0.mlp.")}
    weights["router.b"] = 2.0 * weights["router.b"]
    x = torch.randn(tokens, width, generator=gen).to(torch.bfloat16)
    extra = torch.randn(tokens, width, generator=gen)
    full = {"l0.mlp." + k: v.double() for k, v in weights.items()}
    want = pl.routed_feed_forward(x.double(), full, "l0.mlp.", mlp) + extra.double()
    logits = (x.double() @ weights["router"].double().T + weights["router.b"].double()).sort(dim=-1, descending=True).values
    clear = (logits[:, top - 1] - logits[:, top]) > 5e-3
    assert int(clear.sum()) >= tokens // 2
    names = (("gate_proj.weight", "gate"), ("up_proj.weight", "up"), ("down_proj.weight", "down"))
    spec = RoutedMLPSpec(width, experts, top, GatedMLPSpec(width, ff, "silu", rename=names), score="softmax", renormalise=True,
                         weight_on="output", router_bias=True)
    ctx = BuildContext(dtype=dtype, device=torch.device("cuda"), status=status_word())
    part = build_part(spec, {k: v.to(dtype).cuda() for k, v in weights.items()}, ctx)
    for _ in range(2):      # the second call finds the counts as the first left them
        got = part.forward(x.to(dtype).cuda(), add=extra.cuda()).float().cpu()
    assert int(ctx.status.item()) == 0 and int(part.counts.abs().sum()) == 0
    tol = 1e-4 if dtype == torch.float32 else 3e-2
    assert float((got[clear] - want[clear].float()).abs().max()) <= tol * max(1.0, float(want.abs().max()))


def test_norm_pair_kernel():
    from forge_engine_b200.ops import native

    gen = torch.Generator().manual_seed(1)
    for width in (20, 192, 2560):
        a, b, wa, wb = (torch.randn(*s, generator=gen) for s in ((7, width), (7, width), (width,), (width,)))
        out = torch.empty(7, width, device="cuda")
        native.norm_pair(a.cuda(), b.cuda(), wa.cuda(), wb.cuda(), out, 1e-4, 0.5)
        want = 0.5 * (pl.rms(a.double(), 1e-4) * wa + pl.rms(b.double(), 1e-4) * wb)
        assert float((out.cpu() - want).abs().max()) <= 1e-5


# -- generation through the engine's own entry points ------------------------------------------------
def test_greedy_generation_through_engine_and_scheduler(tmp_path):
    from forge_engine_b200.config import EngineConfig, SchedulerConfig
    from forge_engine_b200.engine import Engine

    cfg = mixed_config()
    weights = write_model(tmp_path / "m", cfg, 18)
    prompts = [tokens_of(cfg, n, 20 + n) for n in (3, 26, 11, 1, 17)]
    engine = Engine.from_pretrained(
        tmp_path / "m",
        engine_config=EngineConfig(max_new_tokens=7, dtype="float32"),
        scheduler_config=SchedulerConfig(max_requests=3, max_batch_size=3, token_budget=12, block_size=4,
                                         block_capacity=96, chunk_size=8),
    )
    outputs = engine.generate(prompts)
    engine.runner.cache.check_consistency()
    assert engine.runner.cache.live_requests == 0
    for prompt, output in zip(prompts, outputs):
        assert len(output) == 7
        ids = list(prompt)
        for token in output:
            ref = oracle(cfg, weights, ids)[-1]
            top = torch.topk(ref, 2).values
            assert token == int(ref.argmax()) or float(top[0] - top[1]) < 1e-3
            ids.append(token)


def test_generate_command(tmp_path, capsys):
    from forge_engine_b200.cli import main

    cfg = pl.config([pl.wkv_layer(), pl.parallel_layer(mlp=None), pl.delta_layer()], loop=(0, 2, 2))
    weights = write_model(tmp_path / "m", cfg, 19)
    prompt = tokens_of(cfg, 9, 1)
    code = main(["generate", "--model", str(tmp_path / "m"), "--prompt-ids", ",".join(map(str, prompt)),
                 "--max-new-tokens", "4", "--dtype", "float32", "--block-size", "4", "--block-capacity", "32"])
    assert code == 0
    printed = [int(t) for t in capsys.readouterr().out.strip().splitlines()[-1].split(",")]
    assert printed == pl.greedy_generate(cfg, weights, prompt, 4)


def test_random_weights_model_steps():
    """Seeded random weights for a configuration (what the benchmark uses; the rank of the decay's
    matrices is then given as ``rank``): logits do not depend on how the prompt was cut."""
    from forge_engine_b200.engine import ModelRunner

    cfg = mixed_config("bfloat16")
    for layer in cfg["layers"]:
        if layer["type"] == "wkv":
            layer["mixer"] = dict(layer["mixer"], rank=12)
    runner = ModelRunner.from_random(cfg, 5, dtype="bfloat16", page_size=16, num_pages=32, max_requests=2, std=0.05)
    tokens = tokens_of(cfg, 140, 3)
    whole = run_schedule(runner, {"a": tokens}, [[("a", 140)]])["a"]
    cut = run_schedule(runner, {"b": tokens}, [[("b", 23)], [("b", 116)], [("b", 1)]])["b"]
    assert torch.isfinite(whole).all()
    assert float((whole - cut).abs().max()) <= 0.05 * max(1.0, float(whole.abs().max()))
