"""The Lozezen design in the engine against the plain implementation of ``plain_lozezen.py``: every
mechanism alone, whole prompts against portions and token-by-token decoding, unequal batches, reused
pages and slots, loud keys just inside and just outside windows and chunks, tokens far back that reach
late logits through the states, the first tokens of a sequence, other sizes, the kernels alone,
generation."""

from __future__ import annotations

import json
import math

import pytest
import torch
from safetensors.torch import save_file

import plain_lozezen as pl

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


def differs(a: torch.Tensor, b: torch.Tensor) -> float:
    return float(((a - b) ** 2).mean().sqrt() / (a**2).mean().sqrt())


oracle = pl.forward


def mixed_config():
    """All mechanisms in one model, the layers' head counts and sizes all different, two layers
    without a feed-forward."""
    return pl.config([
        pl.rglru_layer(width=48, blocks=3, conv=3),
        pl.attention_layer(heads=4, kv_heads=2, size=20),
        pl.rglru_layer(width=64, blocks=2, conv=4, mlp=None),
        pl.parallel_layer(),
        pl.attention_layer(heads=3, kv_heads=1, dim=24, vdim=24, size=33, rot_dims=24, factor=None, mlp=None),
    ])


# -- every mechanism alone --------------------------------------------------------------------
SINGLE = {
    "rglru": [pl.rglru_layer(mlp=None)],
    "rglru_dense": [pl.rglru_layer()],
    "rglru_one_block": [pl.rglru_layer(width=40, blocks=1, mlp=None)],
    "rglru_four_taps": [pl.rglru_layer(width=96, blocks=4, conv=4, mlp=None)],
    "rglru_one_tap": [pl.rglru_layer(conv=1, mlp=None)],
    "rglru_nine_taps": [pl.rglru_layer(conv=9, mlp=None)],
    "rglru_odd": [pl.rglru_layer(width=35, blocks=5, conv=2, mlp=None)],
    "rglru_blocks_of_one": [pl.rglru_layer(width=12, blocks=12, conv=4, mlp=None)],
    "rglru_blocks_of_80": [pl.rglru_layer(width=160, blocks=2, conv=4, mlp=None)],
    "rglru_blocks_of_130": [pl.rglru_layer(width=260, blocks=2, conv=4, mlp=None)],
    "attention": [pl.attention_layer(mlp=None)],
    "attention_dense": [pl.attention_layer()],
    "attention_plain_frequencies": [pl.attention_layer(factor=None, mlp=None)],
    "attention_equal_sizes": [pl.attention_layer(dim=16, vdim=16, rot_dims=16, mlp=None)],
    "attention_odd_sizes": [pl.attention_layer(heads=3, kv_heads=3, dim=10, vdim=26, rot_dims=6, mlp=None)],
    "attention_window_of_one": [pl.attention_layer(size=1, mlp=None)],
    "attention_window_wider_than_the_prompt": [pl.attention_layer(size=500, mlp=None)],
    "attention_heads_of_64": [pl.attention_layer(heads=4, kv_heads=2, dim=64, vdim=64, size=50, rot_dims=64, mlp=None)],
    "attention_heads_of_128": [pl.attention_layer(heads=2, kv_heads=1, dim=128, vdim=128, size=70, rot_dims=32, mlp=None)],
    "parallel": [pl.parallel_layer(mlp=None)],
    "parallel_dense": [pl.parallel_layer()],
    "parallel_left_only": [pl.parallel_layer(right_scale=0.0, mlp=None)],
    "parallel_right_only": [pl.parallel_layer(left_scale=0.0, mlp=None)],
    "parallel_odd_sizes": [pl.parallel_layer(pl.chunk_side(heads=3, kv_heads=3, dim=9, vdim=14, size=7),
                                             pl.retention_side(heads=2, dim=7, vdim=11, rot_dims=4), mlp=None)],
    "parallel_chunks_of_one": [pl.parallel_layer(pl.chunk_side(size=1), mlp=None)],
    "parallel_one_long_chunk": [pl.parallel_layer(pl.chunk_side(size=1000), mlp=None)],
    "parallel_heads_of_64": [pl.parallel_layer(pl.chunk_side(heads=4, kv_heads=2, dim=64, vdim=64, size=48),
                                               pl.retention_side(heads=2, dim=64, vdim=64, rot_dims=64), mlp=None)],
    "parallel_heads_of_128": [pl.parallel_layer(pl.chunk_side(heads=2, kv_heads=2, dim=128, vdim=128, size=96),
                                                pl.retention_side(heads=1, dim=96, vdim=128, rot_dims=32), mlp=None)],
    "parallel_decays_of_one_and_zero": [pl.parallel_layer(right=pl.retention_side(heads=4, decay=[1.0, 0.0, 0.5, 0.999]), mlp=None)],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_each_mechanism_alone(tmp_path, name, dtype):
    """A whole prompt longer than a tile or chunk of the recurrences, then the same cut into a short
    portion, a long one and single tokens."""
    cfg = pl.config(SINGLE[name])
    weights = write_model(tmp_path / "m", cfg, 11)
    tokens = tokens_of(cfg, 137, 5)
    runner = make_runner(tmp_path / "m", dtype)
    want = oracle(cfg, weights, tokens)
    whole = run_schedule(runner, {"a": tokens}, [[("a", 137)]])["a"]
    cut = run_schedule(runner, {"b": tokens}, [[("b", 2)], [("b", 19)], [("b", 107)]] + [[("b", 1)] for _ in range(9)])["b"]
    assert_close(whole, want, dtype, name)
    assert_close(cut, want, dtype, name + ", cut")


def test_residual_after_every_layer(tmp_path):
    """The residual stream after every layer, in 32-bit, against the plain implementation."""
    from forge_engine_b200.engine import StepEntry

    cfg = mixed_config()
    weights = write_model(tmp_path / "m", cfg, 12)
    tokens = tokens_of(cfg, 45, 6)
    want = []
    pl.forward(cfg, weights, tokens, layers_out=want)
    runner = make_runner(tmp_path / "m", "float32", use_graphs=False)
    seen = []
    for block in runner.model.blocks:
        inner = block.forward

        def spy(h, pending, batch, cache, inner=inner):
            update, norm = inner(h, pending, batch, cache)
            seen.append((h + pl.rms(update.float(), norm.eps) * norm.weight).cpu())
            return update, norm

        block.forward = spy
    runner.begin("a")
    runner.step([StepEntry("a", tokens, [len(tokens) - 1])])
    runner.check_status()
    assert len(seen) == len(want) == 5
    for index, (got, ref) in enumerate(zip(seen, want)):
        assert float((got - ref.float()).abs().max()) <= 2e-4 * max(1.0, float(ref.abs().max())), f"layer {index}"


# -- the same sequence cut in different ways ------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
def test_prefill_against_token_by_token_decoding(tmp_path, dtype):
    cfg = mixed_config()
    weights = write_model(tmp_path / "m", cfg, 13)
    tokens = tokens_of(cfg, 45, 7)
    runner = make_runner(tmp_path / "m", dtype)
    ref = oracle(cfg, weights, tokens)
    whole = run_schedule(runner, {"a": tokens}, [[("a", 45)]])["a"]
    single = run_schedule(runner, {"b": tokens}, [[("b", 1)] for _ in range(45)])["b"]
    assert_close(whole, ref, dtype, "whole prompt")
    assert_close(single, ref, dtype, "token by token")


# around the tiles and chunks of 64 tokens, the 96 from which on a portion runs in chunks, the windows of
# 20 and 33 and the chunks of 18
SIZES = ((7, 2, 13, 3, 2, 5, 1, 16, 2, 9), (2,) * 20, (1, 2, 1, 3, 30, 2), (95, 2, 96, 3), (97, 64, 65, 1, 2), (128, 129, 2), (63, 1, 192, 4),
         (17, 2, 16, 1, 18, 36, 2), (20, 19, 21, 33, 2, 32, 34), (160, 2, 2, 100))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", SIZES)
def test_portions_of_several_sizes(tmp_path, sizes, dtype):
    """Portions down to two tokens (and one), cut in the middle of pages, windows and chunks, at their
    borders and one token beside them."""
    cfg = mixed_config()
    weights = write_model(tmp_path / "m", cfg, 14)
    tokens = tokens_of(cfg, sum(sizes), 8)
    runner = make_runner(tmp_path / "m", dtype)
    got = run_schedule(runner, {"a": tokens}, [[("a", n)] for n in sizes])["a"]
    assert_close(got, oracle(cfg, weights, tokens), dtype, f"portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch_against_each_alone(tmp_path, dtype):
    cfg = mixed_config()
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
    """Entries whose chunks lie side by side in the scratch, none a multiple of a chunk; tiles of the
    gated recurrence that hold the end of one entry and the start of another."""
    cfg = mixed_config()
    weights = write_model(tmp_path / "m", cfg, 35)
    requests = {"a": tokens_of(cfg, 150, 1), "b": tokens_of(cfg, 203, 2), "c": tokens_of(cfg, 97, 3), "d": tokens_of(cfg, 5, 4)}
    runner = make_runner(tmp_path / "m", dtype, num_pages=160)
    got = run_schedule(runner, requests, [[("d", 3), ("a", 99), ("b", 131), ("c", 96)], [("b", 72), ("d", 2), ("c", 1), ("a", 51)]])
    for key, tokens in requests.items():
        assert_close(got[key], oracle(cfg, weights, tokens), dtype, f"request {key}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_slots_freed_and_used_again(tmp_path, dtype):
    """Two slots and a small pool: later requests get the pages and the states of earlier ones,
    which must read as new (every state: the recurrences', the convolution's inputs)."""
    cfg = mixed_config()
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
def test_long_decoding_in_fewer_pages_than_tokens(tmp_path, dtype):
    """A short prompt, then more single tokens than windows and chunks hold: their pages are given back
    and used again by the same request.  The steps are replayed from captured graphs."""
    cfg = mixed_config()
    weights = write_model(tmp_path / "m", cfg, 17)
    tokens = tokens_of(cfg, 150, 9)
    runner = make_runner(tmp_path / "m", dtype, page_size=4, num_pages=11)
    got = run_schedule(runner, {"a": tokens}, [[("a", 5)]] + [[("a", 1)] for _ in range(145)])["a"]
    assert_close(got, oracle(cfg, weights, tokens), dtype, "long decoding")
    assert runner.use_graphs and runner.graphs.captured


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", (16, 100))
def test_mixed_steps_replayed_from_graphs(tmp_path, portion, dtype):
    """Steps that bring a prompt portion beside two decoding requests, captured at first sight
    and replayed (filler entries pad them to their bucket).  Logits at every entry's last token."""
    from forge_engine_b200.engine import StepEntry

    cfg = mixed_config()
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
    earlier request's keys and states: no earlier inputs of the convolution, states of zero."""
    cfg = mixed_config()
    weights = write_model(tmp_path / "m", cfg, 25)
    runner = make_runner(tmp_path / "m", dtype, max_requests=4, num_pages=24)
    warm = {key: tokens_of(cfg, 12, 40 + i) for i, key in enumerate("wxyz")}
    run_schedule(runner, warm, [[(key, 12) for key in warm]])
    requests = {key: tokens_of(cfg, n, 30 + n) for key, n in (("a", 1), ("b", 2), ("c", 3), ("d", 5))}
    got = run_schedule(runner, requests, [[("a", 1), ("b", 1), ("c", 3), ("d", 2)], [("b", 1), ("d", 3)]])
    for key, tokens in requests.items():
        assert_close(got[key], oracle(cfg, weights, tokens), dtype, f"request {key}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_decoding_requests(tmp_path, dtype):
    """More entries than a tile of the one-launch step holds."""
    cfg = pl.config([pl.rglru_layer(width=80, blocks=2, conv=4), pl.parallel_layer(mlp=None)])
    weights = write_model(tmp_path / "m", cfg, 27)
    requests = {f"r{i}": tokens_of(cfg, 4 + i % 3, 50 + i) for i in range(21)}
    runner = make_runner(tmp_path / "m", dtype, max_requests=21, num_pages=64)
    schedule = [[(key, 3) for key in requests], [(key, 1) for key in requests]]
    schedule += [[(key, 1) for key, tokens in requests.items() if len(tokens) > n] for n in (4, 5)]
    got = run_schedule(runner, requests, schedule)
    for key, tokens in requests.items():
        assert_close(got[key], oracle(cfg, weights, tokens), dtype, f"request {key}")


# -- other sizes ------------------------------------------------------------------------------
OTHER = {
    "narrow": dict(layers=[pl.rglru_layer(width=4, blocks=1, conv=2, mlp=None), pl.attention_layer(heads=1, kv_heads=1, dim=2, vdim=3, rot_dims=2, size=5, mlp=pl.dense(8)),
                           pl.parallel_layer(pl.chunk_side(heads=1, kv_heads=1, dim=4, vdim=2, size=9),
                                             pl.retention_side(heads=1, dim=4, vdim=4, rot_dims=2), mlp=None)], width=20, vocab=11),
    "width_not_in_eights": dict(layers=[pl.rglru_layer(width=36), pl.attention_layer(), pl.parallel_layer()], width=36),
    "recurrence_wider_than_the_stream": dict(layers=[pl.rglru_layer(width=200, blocks=5, conv=4), pl.rglru_layer(width=24, blocks=2)], width=48),
    "every_head_its_own_keys": dict(layers=[pl.attention_layer(heads=4, kv_heads=None), pl.parallel_layer(pl.chunk_side(heads=4, kv_heads=None))]),
    "many_heads_per_key_head": dict(layers=[pl.attention_layer(heads=12, kv_heads=1, dim=8, vdim=8, rot_dims=4, mlp=None),
                                            pl.parallel_layer(pl.chunk_side(heads=12, kv_heads=1, dim=8, vdim=8), mlp=None)]),
    "many_state_heads": dict(layers=[pl.parallel_layer(right=pl.retention_side(heads=16, dim=8, vdim=8), mlp=None)]),
    "wide_heads": dict(layers=[pl.parallel_layer(right=pl.retention_side(heads=1, dim=128, vdim=256, rot_dims=128), mlp=None)], width=96),
    "wider_heads": dict(layers=[pl.parallel_layer(right=pl.retention_side(heads=1, dim=200, vdim=320, rot_dims=2), mlp=None)], width=96),
    "scale_one_eps_large": dict(layers=[pl.attention_layer(scale=1.0), pl.rglru_layer(), pl.parallel_layer(pl.chunk_side(scale=1.0))], eps=0.5),
    "ones": dict(layers=[pl.parallel_layer(left_scale=1.0, right_scale=1.0), pl.attention_layer(factor=1.0), pl.rglru_layer(width=9, blocks=1, conv=1)], scale=1.0),
    "equal_decays": dict(layers=[pl.parallel_layer(right=pl.retention_side(decay=[0.9, 0.9, 0.9]))]),
    "base_of_one": dict(layers=[pl.attention_layer(base=1.0)]),
    "one_kind_only": dict(layers=[pl.rglru_layer(mlp=None), pl.rglru_layer(), pl.rglru_layer(mlp=None)]),
    "window_and_chunk_of_a_page": dict(layers=[pl.attention_layer(size=8), pl.parallel_layer(pl.chunk_side(size=8))]),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(OTHER))
def test_other_sizes_and_values_that_are_one_or_equal(tmp_path, name, dtype):
    options = dict(OTHER[name])
    cfg = pl.config(options.pop("layers"), **options)
    weights = write_model(tmp_path / "m", cfg, 21)
    tokens = tokens_of(cfg, 140, 10)
    runner = make_runner(tmp_path / "m", dtype, page_size=8, num_pages=48)
    ref = oracle(cfg, weights, tokens)
    whole = run_schedule(runner, {"a": tokens}, [[("a", 140)]])["a"]
    cut = run_schedule(runner, {"b": tokens}, [[("b", 19)], [("b", 2)], [("b", 101)], [("b", 2)]] + [[("b", 1)] for _ in range(16)])["b"]
    assert_close(whole, ref, dtype, name)
    assert_close(cut, ref, dtype, name + ", cut")


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_of_the_tensor_core_paths(tmp_path, dtype):
    """Sizes in sixteens, so that the bfloat16 engine takes its tensor-core products and all
    tensor-core attention kernels, with steps long enough for several row tiles and key tiles."""
    cfg = pl.config([pl.rglru_layer(width=256, blocks=2, conv=4, mlp=pl.dense(128)),
                     pl.attention_layer(heads=4, kv_heads=2, dim=64, vdim=64, rot_dims=32, size=150, mlp=pl.dense(128)),
                     pl.parallel_layer(pl.chunk_side(heads=4, kv_heads=2, dim=64, vdim=64, size=170),
                                       pl.retention_side(heads=2, dim=32, vdim=64, rot_dims=32), mlp=None),
                     pl.attention_layer(heads=6, kv_heads=2, dim=64, vdim=32, rot_dims=64, size=90, mlp=None),
                     pl.parallel_layer(pl.chunk_side(heads=2, kv_heads=1, dim=128, vdim=128, size=256),
                                       pl.retention_side(heads=2, dim=64, vdim=64, rot_dims=16), mlp=None)], width=128)
    weights = write_model(tmp_path / "m", cfg, 22)
    tokens = tokens_of(cfg, 400, 11)
    runner = make_runner(tmp_path / "m", dtype, page_size=16, num_pages=64)
    ref = oracle(cfg, weights, tokens)
    whole = run_schedule(runner, {"a": tokens}, [[("a", 400)]])["a"]
    cut = run_schedule(runner, {"b": tokens}, [[("b", 130)], [("b", 2)], [("b", 200)], [("b", 63)]] + [[("b", 1)] for _ in range(5)])["b"]
    assert_close(whole, ref, dtype, "whole")
    assert_close(cut, ref, dtype, "cut")


# -- loud keys at the edges of windows and chunks -----------------------------------------------------
def loud_pair(cfg: dict, weights: dict, key_token: int, query_token: int, wish: float) -> None:
    """Make the key of ``key_token`` point where the query of ``query_token`` points in every head
    of the first layer's softmax attention, and set the score scale so that the pair's score is ``wish``
    in the weakest head: that key then takes nearly all of that query's weight."""
    kind = cfg["layers"][0]["type"]
    m, p = (cfg["layers"][0]["mixer"], "l0.mix.") if kind == "attention" else (cfg["layers"][0]["mixer"]["left"], "l0.mix.left.")
    heads, kv_heads, dim, eps = m["heads"], m["kv_heads"], m["dim"], cfg["norm"]["eps"]
    rot = m["rot"]["dims"] if kind == "attention" else 0
    w = {k: v.double() for k, v in weights.items()}
    row = lambda token: pl.norm_around_one(w["embed"][token] * cfg["embedding"]["scale"], w["l0.norm1"], eps)  # noqa: E731

    def head_rows(name, token, count):
        x = (w[p + name] @ row(token) + w[f"{p}{name}.b"]).view(count, dim)
        return x if kind == "attention" else pl.rms(x, eps) * w[f"{p}{name}.norm"]

    query = head_rows("q", query_token, heads).view(kv_heads, heads // kv_heads, dim)
    target = query.mean(dim=1)
    target[:, :rot] = 0.0                                    # the rotated elements turn with the distance
    if kind != "attention":
        target = target / w[p + "k.norm"]
    h = torch.linalg.lstsq(w[p + "k"], target.reshape(-1)[:, None]).solution[:, 0]
    embed = h / (1.0 + w["l0.norm1"])
    weights["embed"][key_token] = (embed / embed.pow(2).mean().sqrt() / cfg["embedding"]["scale"]).to(weights["embed"].dtype)
    w["embed"] = weights["embed"].double()
    score = (query[:, :, rot:] * head_rows("k", key_token, kv_heads)[:, None, rot:]).sum(-1)
    assert float(score.min()) > 0
    m["scale"] = wish / float(score.min())


QUIET = pl.retention_side(heads=2, dim=8, vdim=8, decay=[0.0, 0.0])      # remembers nothing
EDGES = {
    "window_plain_kernel": pl.attention_layer(heads=4, kv_heads=2, dim=24, vdim=20, size=37, rot_dims=2, base=1e6, mlp=None),
    "window_tensor_cores": pl.attention_layer(heads=4, kv_heads=2, dim=32, vdim=16, size=75, rot_dims=4, base=1e6, mlp=None),
    "window_heads_of_64": pl.attention_layer(heads=2, kv_heads=1, dim=64, vdim=64, size=130, rot_dims=4, base=1e6, factor=None, mlp=None),
    "window_heads_of_128": pl.attention_layer(heads=2, kv_heads=1, dim=128, vdim=128, size=100, rot_dims=8, base=1e6, mlp=None),
    "chunk_plain_kernel": pl.parallel_layer(pl.chunk_side(heads=4, kv_heads=2, dim=20, vdim=12, size=37), QUIET, right_scale=0.05, mlp=None),
    "chunk_tensor_cores": pl.parallel_layer(pl.chunk_side(heads=4, kv_heads=2, dim=32, vdim=48, size=75), QUIET, right_scale=0.05, mlp=None),
    "chunk_heads_of_64": pl.parallel_layer(pl.chunk_side(heads=2, kv_heads=1, dim=64, vdim=64, size=130), QUIET, right_scale=0.05, mlp=None),
    "chunk_heads_of_128": pl.parallel_layer(pl.chunk_side(heads=2, kv_heads=1, dim=128, vdim=128, size=100), QUIET, right_scale=0.05, mlp=None),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", sorted(EDGES))
def test_a_loud_key_just_inside_and_just_outside(tmp_path, kind, dtype):
    """One layer, one key that takes nearly all the weight of every loud query that sees it: for windows
    at distance size - 1 (the last one seen) and size, for chunks at the first position of the query's
    chunk and the one before, and at page borders; in a prompt's own portion, in later portions and in
    decoding, queries at the first and last position of a chunk."""
    cfg = pl.config([EDGES[kind]], width=192, vocab=40)
    layer = cfg["layers"][0] = json.loads(json.dumps(EDGES[kind]))
    key_token, query_token = 38, 39

    def change(weights):
        loud_pair(cfg, weights, key_token, query_token, 22.0)

    change(pl.random_weights(cfg, 23))            # sets the scale in cfg before the folder is written
    weights = write_model(tmp_path / "m", cfg, 23, change=change)
    length = 330
    runner = make_runner(tmp_path / "m", dtype, page_size=16, num_pages=64)
    if layer["type"] == "attention":
        size = layer["mixer"]["mask"]["size"]
        cases = [(at, [(at + 1, True), (at + size - 1, True), (at + size, False), (at + size + 1, False)])
                 for at in (0, 15, 16, 127, 128, 321 - size)]
    else:
        size = layer["mixer"]["left"]["mask"]["size"]
        cases = []
        for c in (0, 1, 320 // size - 1):
            first = c * size
            cases.append((first, [(first + 1, True), (first + size - 1, True), (first + size, False), (first + size + 7, False)]))
            cases.append((first + size - 1, [(first + size, False), (first + 2 * size - 1, False)]))
    for at, queries in cases:
        tokens = tokens_of(cfg, length, 12, avoid=(key_token, query_token))
        queries = [(q, sees) for q, sees in queries if at < q < length]
        plain = list(tokens)
        for q, _ in queries:
            tokens[q] = plain[q] = query_token
        tokens[at] = key_token
        ref, without = oracle(cfg, weights, tokens), oracle(cfg, weights, plain)
        for q, sees in queries:
            if sees:
                assert differs(ref[q], without[q]) > 0.2, f"the key at {at} decides the logits at {q}"
            else:
                assert differs(ref[q], without[q]) < 1e-9, f"the key at {at} is not seen at {q}"
        whole = run_schedule(runner, {"a": tokens}, [[("a", length)]])["a"]
        single = 14 if at < 200 else 50
        cut = run_schedule(runner, {"b": tokens}, [[("b", at + 1)], [("b", 2)], [("b", length - at - 3 - single)]] + [[("b", 1)] for _ in range(single)]
                           if length - at - 3 - single > 0 else [[("b", at + 1)]] + [[("b", 1)] for _ in range(length - at - 1)])["b"]
        for got, what in ((whole, "prompt"), (cut, "cut")):
            assert_close(got, ref, dtype, f"{what}, key at {at}")
            for q, _ in queries:
                assert_close(got[q : q + 1], ref[q : q + 1], dtype, f"{what}, key at {at}, query at {q}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ("window_heads_of_64", "chunk_heads_of_64", "window_plain_kernel", "chunk_tensor_cores"))
def test_a_loud_key_read_by_every_decoded_token(tmp_path, kind, dtype):
    """Every token is decoded on its own and asks for the loud key, until and after it goes out of sight."""
    cfg = pl.config([json.loads(json.dumps(EDGES[kind]))], width=192, vocab=40)
    key_token, query_token = 38, 39

    def change(weights):
        loud_pair(cfg, weights, key_token, query_token, 22.0)

    change(pl.random_weights(cfg, 24))
    weights = write_model(tmp_path / "m", cfg, 24, change=change)
    tokens = tokens_of(cfg, 20, 3, avoid=(key_token, query_token)) + [key_token] + [query_token] * 150
    runner = make_runner(tmp_path / "m", dtype, page_size=16, num_pages=16)
    ref = oracle(cfg, weights, tokens)
    got = run_schedule(runner, {"a": tokens}, [[("a", 19)]] + [[("a", 1)] for _ in range(152)])["a"]
    assert_close(got, ref, dtype, kind)
    for q in range(21, 171):
        assert_close(got[q : q + 1], ref[q : q + 1], dtype, f"{kind}, token {q}")


# -- far tokens through the states ----------------------------------------------------------------------
def slow_decay(weights: dict) -> None:
    for name, t in weights.items():
        if name.endswith(".lam"):
            weights[name] = torch.full_like(t, -9.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ("rglru", "rglru_large", "retention"))
def test_a_token_far_back_reaches_late_logits_through_the_state(tmp_path, kind, dtype):
    """States that hardly decay: a token changed at the start, at tile and chunk borders or beside them
    moves the logits hundreds of tokens later, in prompts, in later portions and in decoding."""
    layer = {"rglru": pl.rglru_layer(width=32, blocks=2, conv=4, mlp=None), "rglru_large": pl.rglru_layer(width=192, blocks=2, conv=4, mlp=None),
             "retention": pl.parallel_layer(pl.chunk_side(size=5), pl.retention_side(heads=2, dim=32, vdim=32, rot_dims=8, decay=[0.9995, 1.0]),
                                            mlp=None)}[kind]
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


# -- kernels alone -------------------------------------------------------------------------------
def entry_tensors(counts: list):
    cu = [0]
    for n in counts:
        cu.append(cu[-1] + n)
    entry = [e for e, n in enumerate(counts) for _ in range(n)]
    make = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")  # noqa: E731
    return make(cu), make(entry), make(list(range(len(counts)))[::-1])      # slots in reverse order of the entries


def status_word():
    return torch.zeros(1, dtype=torch.int32, device="cuda")


COUNTS = ([1, 1, 1], [1] * 19, [5, 1, 95], [96, 3, 130], [200], [63, 2, 1, 64, 1, 1])


@pytest.mark.parametrize("weights", (torch.float32, torch.bfloat16))
@pytest.mark.parametrize("counts", COUNTS, ids=str)
@pytest.mark.parametrize("blocks, part, taps", ((1, 16, 4), (3, 5, 1), (2, 27, 2), (2, 64, 4), (2, 80, 4), (1, 200, 3), (2, 264, 4), (1, 520, 9)))
def test_rglru_kernels(blocks, part, taps, counts, weights):
    """From states that are not zero; decays from exactly 1 (rate 0) to exactly 0."""
    from forge_engine_b200.ops import native

    gen = torch.Generator().manual_seed(part + taps)
    rand = lambda *shape: torch.randn(*shape, generator=gen, dtype=torch.float64)  # noqa: E731
    n, width = sum(counts), blocks * part
    proj, conv, conv_bias = rand(n, 2 * width), 0.6 * rand(width, taps), 0.5 * rand(width)
    bias, sums = 0.7 * rand(2 * width), proj
    proj = sums + bias
    w = [(rand(blocks, part, part) * 1.5 / math.sqrt(part)).to(torch.bfloat16).double() for _ in range(2)]
    b = [0.5 * rand(width) for _ in range(2)]
    rate = -torch.exp(3.0 * rand(width) - 3.0)
    rate[::7], rate[3::7] = 0.0, -1e4
    state, history = rand(len(counts) + 1, width), rand(len(counts) + 1, taps - 1, width)
    cu, entry, slots = entry_tensors(counts)
    want, want_state, want_history = torch.empty(n, width, dtype=torch.float64), state.clone(), history.clone()
    for e in range(len(counts)):
        s = int(slots[e])
        rows = torch.cat([history[s], proj[cu[e] : cu[e + 1], width:]])
        u = sum(rows[j : j + counts[e]] * conv[:, j] for j in range(taps)) + conv_bias
        r, i = (pl.sigmoid(torch.einsum("tbk,bok->tbo", u.view(-1, blocks, part), w[g]).flatten(1) + b[g]) for g in range(2))
        log_a = rate * r
        write = torch.sqrt(-torch.expm1(2 * log_a)) * i * u
        for t in range(counts[e]):
            want_state[s] = torch.exp(log_a[t]) * want_state[s] + write[t]
            want[cu[e] + t] = want_state[s] * pl.gelu_tanh(proj[cu[e] + t, :width])
        want_history[s] = rows[len(rows) - (taps - 1):]
    dev = lambda t: t.float().cuda().contiguous()  # noqa: E731
    got_state, got_history, out, status = dev(state), dev(history), torch.empty(n, width, device="cuda"), status_word()
    native.rglru(dev(sums), 0, width, dev(conv.T), dev(conv_bias), w[0].to(weights).cuda(), w[1].to(weights).cuda(), dev(bias[:width]),
                 dev(bias[width:]), dev(b[0]), dev(b[1]), dev(rate), got_state, got_history if taps > 1 else None, slots, cu, entry, out, len(counts), max(counts), status)
    assert int(status.item()) == 0 and not native.damaged_canaries()
    tol = 2e-5 if weights == torch.float32 else 1e-4        # u as a sum of two bfloat16 numbers
    assert float((out.cpu() - want).abs().max()) <= tol * max(1.0, float(want.abs().max()))
    assert float((got_state.cpu() - want_state).abs().max()) <= tol * max(1.0, float(want_state.abs().max()))
    if taps > 1:
        assert float((got_history.cpu() - want_history).abs().max()) <= 1e-6 * float(want_history.abs().max())


@pytest.mark.parametrize("counts", COUNTS, ids=str)
@pytest.mark.parametrize("interleaved", (False, True))
@pytest.mark.parametrize("heads, dk, dv, rot", ((2, 8, 8, 8), (3, 12, 20, 6), (1, 64, 64, 64), (2, 48, 64, 2), (1, 128, 256, 0), (1, 100, 36, 40), (1, 256, 320, 16), (2, 33, 7, 32)))
def test_retention_kernels(heads, dk, dv, rot, interleaved, counts):
    """Decays of 1, 0 and in between, from states that are not zero; rotated in the walk or, for steps with
    long portions, beforehand; with and without a weight of the norm."""
    from forge_engine_b200.ops import native

    gen = torch.Generator().manual_seed(dk * 7 + dv)
    rand = lambda *shape: torch.randn(*shape, generator=gen, dtype=torch.float64)  # noqa: E731
    n = sum(counts)
    q, k, v, gate = rand(n, heads, dk), rand(n, heads, dk), rand(n, heads, dv), rand(n, heads, dv)
    decay = torch.tensor([0.96, 0.0, 1.0][:heads], dtype=torch.float64)
    angle = 3.0 * rand(n, max(rot // 2, 1))
    state = 0.5 * rand(len(counts) + 1, heads, dk, dv)
    norm = 1 + 0.1 * rand(dv) if dk % 8 == 0 else None

    def turned(x):
        if rot == 0:
            return x
        head = x[..., :rot]
        a, b = (head[..., 0::2], head[..., 1::2]) if interleaved else (head[..., : rot // 2], head[..., rot // 2 :])
        c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
        pair = (a * c - b * s, b * c + a * s)
        head = torch.stack(pair, dim=-1).flatten(-2) if interleaved else torch.cat(pair, dim=-1)
        return torch.cat([head, x[..., rot:]], dim=-1)

    cu, _, slots = entry_tensors(counts)
    qr, kr = turned(q), turned(k) * dk**-0.5
    want, want_state = torch.empty(n, heads, dv, dtype=torch.float64), state * dk**-0.5      # the engine's state holds unscaled keys
    for e in range(len(counts)):
        for h in range(heads):
            S = want_state[slots[e], h]
            for t in range(cu[e], cu[e + 1]):
                S.copy_(decay[h] * S + torch.outer(kr[t, h], v[t, h]))
                want[t, h] = S.T @ qr[t, h]
    raw = want
    want = (pl.rms(want, 1e-5) * (1.0 if norm is None else norm) * pl.silu(gate)).view(n, heads * dv)
    long = max(counts) >= native.state_long_from()
    dev = lambda t: t.float().cuda().contiguous()  # noqa: E731
    proj = dev(torch.cat([x.reshape(n, -1) for x in ((qr, kr * dk**0.5) if long else (q, k)) + (v, gate)], dim=1))
    table = None if long or rot == 0 else dev(torch.stack([torch.cos(angle), torch.sin(angle)], dim=-1))
    sizes = [heads * dk, heads * dk, heads * dv]
    got_state, out, status = dev(state), torch.empty(n, heads * dv, device="cuda"), status_word()
    native.retention(proj, [sum(sizes[:j]) for j in range(4)], dk**-0.5, dev(decay), table, rot, interleaved, None if norm is None else dev(norm),
                     1e-5, got_state, slots, cu, out, len(counts), max(counts), status)
    assert int(status.item()) == 0 and not native.damaged_canaries()
    # rows whose output nearly cancels are divided by a tiny root mean square: compare where it is not tiny
    clear = (raw.pow(2).mean(-1) > 1e-4).repeat_interleave(dv, dim=1).view(n, heads * dv)
    assert n < 20 or float(clear.float().mean()) > 0.3
    assert float(((out.cpu() - want).abs() * clear).max()) <= 1e-3 * max(1.0, float(want.abs().max()))
    want_state = want_state * dk**0.5
    assert float((got_state.cpu() - want_state).abs().max()) <= 3e-5 * max(1.0, float(want_state.abs().max()))


@pytest.mark.parametrize("interleaved", (False, True))
@pytest.mark.parametrize("mode", ("none", "before", "after"))
@pytest.mark.parametrize("heads, kv, dim, vdim, rot", ((4, 2, 64, 64, 64), (4, 2, 64, 32, 16), (3, 3, 24, 20, 8), (6, 1, 128, 128, 96), (2, 1, 48, 100, 0),
                                                       (2, 2, 10, 7, 6), (2, 1, 160, 64, 40), (1, 1, 256, 256, 256), (3, 1, 20, 16, 12)))
def test_preparation_of_queries_keys_and_values(heads, kv, dim, vdim, rot, mode, interleaved):
    """Bias, norm per head (before or after the rotation), rotation, pages: by heads in registers where the
    sizes keep to fours, else by heads in shared memory; the queries written where they were read."""
    from forge_engine_b200.ops import native

    gen = torch.Generator().manual_seed(dim + rot)
    rand = lambda *shape: torch.randn(*shape, generator=gen, dtype=torch.float64)  # noqa: E731
    n, page_size, pages = 13, 4, 9
    sizes = [heads * dim, kv * dim, kv * vdim]
    sums, bias = rand(n, sum(sizes)), rand(sum(sizes))
    qw, kw = 1 + 0.2 * rand(dim), 1 + 0.2 * rand(dim)
    angle = 3.0 * rand(n, max(rot // 2, 1))
    positions = torch.tensor(list(range(3, 12)) + list(range(4)), dtype=torch.int32)
    entry = torch.tensor([0] * 9 + [1] * 4, dtype=torch.int32)
    table = torch.tensor([[7, 2, 5], [0, -1, -1]], dtype=torch.int32)

    def turned(x):
        if rot == 0:
            return x
        head = x[..., :rot]
        a, b = (head[..., 0::2], head[..., 1::2]) if interleaved else (head[..., : rot // 2], head[..., rot // 2 :])
        c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
        pair = (a * c - b * s, b * c + a * s)
        return torch.cat([torch.stack(pair, dim=-1).flatten(-2) if interleaved else torch.cat(pair, dim=-1), x[..., rot:]], dim=-1)

    def prepared(x, w):
        if mode == "after":
            return pl.rms(turned(x), 1e-3) * w
        return turned(pl.rms(x, 1e-3) * w) if mode == "before" else turned(x)

    q, k, v = (sums + bias).split(sizes, dim=1)
    want_q, want_k, want_v = prepared(q.reshape(n, heads, dim), qw), prepared(k.reshape(n, kv, dim), kw), v.reshape(n, kv, vdim)
    dev = lambda t: t.float().cuda().contiguous()  # noqa: E731
    proj, k_cache, v_cache, status = dev(sums), torch.zeros(pages, kv, page_size, dim, device="cuda"), torch.zeros(pages, kv, page_size, vdim, device="cuda"), status_word()
    norm = {"none": native.PREP_NORM_NONE, "before": native.PREP_NORM_HEAD, "after": native.PREP_NORM_HEAD_AFTER}[mode]
    ends = (sizes[0], sizes[0] + sizes[1])
    all_bias = dev(bias)
    native.qkv_prepare(
        q=proj[:, : ends[0]], q_heads=heads, q_dim=dim, q_norm=(norm, dim, dev(qw)), q_out=proj, q_out_strides=(sum(sizes), dim),
        k=proj[:, ends[0] : ends[1]], k_heads=kv, k_dim=dim, k_norm=(norm, dim, dev(kw)), v=proj[:, ends[1] :], v_dim=vdim, eps=1e-3,
        table=dev(torch.stack([torch.cos(angle), torch.sin(angle)], dim=-1)) if rot else None, rot_dims=rot, interleaved=interleaved,
        k_cache=k_cache, v_cache=v_cache, block_table=table.cuda(), positions=positions.cuda(), token_entry=entry.cuda(), status=status,
        q_bias=all_bias[: ends[0]], k_bias=all_bias[ends[0] : ends[1]], v_bias=all_bias[ends[1] :])
    assert int(status.item()) == 0
    assert float((proj[:, : ends[0]].cpu().view(n, heads, dim) - want_q).abs().max()) <= 2e-5 * float(want_q.abs().max())
    filled = torch.zeros(pages, page_size, dtype=torch.bool)
    for t in range(n):
        page, slot = int(table[entry[t], positions[t] // page_size]), int(positions[t] % page_size)
        filled[page, slot] = True
        assert float((k_cache[page, :, slot].cpu() - want_k[t]).abs().max()) <= 2e-5 * float(want_k.abs().max())
        assert float((v_cache[page, :, slot].cpu() - want_v[t]).abs().max()) <= 2e-5 * float(want_v.abs().max())
    for cache in (k_cache, v_cache):
        assert float((cache.cpu() * ~filled[:, None, :, None]).abs().max()) == 0.0


def test_weighted_sum_kernel():
    from forge_engine_b200.ops import native

    gen = torch.Generator().manual_seed(1)
    for width in (1, 20, 192, 2561):
        a, b = torch.randn(7, width, generator=gen), torch.randn(7, width, generator=gen)
        out = torch.empty(7, width, device="cuda")
        native.weighted_sum(a.cuda(), b.cuda(), 0.6, -1.25, out)
        assert float((out.cpu().double() - (0.6 * a.double() - 1.25 * b.double())).abs().max()) <= 1e-6


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

    cfg = pl.config([pl.rglru_layer(), pl.parallel_layer(mlp=None), pl.attention_layer()])
    weights = write_model(tmp_path / "m", cfg, 19)
    prompt = tokens_of(cfg, 9, 1)
    code = main(["generate", "--model", str(tmp_path / "m"), "--prompt-ids", ",".join(map(str, prompt)),
                 "--max-new-tokens", "4", "--dtype", "float32", "--block-size", "4", "--block-capacity", "32"])
    assert code == 0
    printed = [int(t) for t in capsys.readouterr().out.strip().splitlines()[-1].split(",")]
    assert printed == pl.greedy_generate(cfg, weights, prompt, 4)


def test_random_weights_model_steps():
    """Seeded random weights for a configuration (what the benchmark uses): logits do not depend on how
    the prompt was cut."""
    from forge_engine_b200.engine import ModelRunner

    cfg = mixed_config()
    runner = ModelRunner.from_random(cfg, 5, dtype="bfloat16", page_size=16, num_pages=32, max_requests=2, std=0.05)
    tokens = tokens_of(cfg, 140, 3)
    whole = run_schedule(runner, {"a": tokens}, [[("a", 140)]])["a"]
    cut = run_schedule(runner, {"b": tokens}, [[("b", 23)], [("b", 116)], [("b", 1)]])["b"]
    assert torch.isfinite(whole).all()
    assert float((whole - cut).abs().max()) <= 0.05 * max(1.0, float(whole.abs().max()))
