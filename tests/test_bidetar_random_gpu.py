"""Bidetar configurations drawn by seed against the plain implementation: head counts and sizes, chunks from one position
to none, rotated shares, bands, feed-forward sizes and none, loops anywhere, the model's constants.  Each draw replays a
mixed trace (portions of prompts beside decoded tokens on few pages and three slots) in float32 and bfloat16."""

from __future__ import annotations

import random

import pytest
import torch
from bidetar_models import as_double, layer, make_config, make_weights, write_folder
from plain_bidetar import forward
from test_kopatar_gpu import DTYPES, _compare, _replay, _runner, _sequences
from trace_tools import mixed, portions, tail_one_by_one, whole

DRAWS = 10


def _bands(rng, original):
    low = rng.choice([0.5, 1.0, 2.0])
    return None if rng.random() < 0.3 else {"factor": rng.choice([2.0, 4.5, 16.0]), "low": low, "high": low * rng.choice([2.0, 4.0, 7.0]),
                                            "original": rng.choice(original)}


def _loop(rng, count):
    if rng.random() < 0.25:
        return None
    start = rng.randint(0, count - 1)
    return start, rng.randint(start + 1, count), rng.randint(1, 3)


def draw_config(seed: int) -> dict:
    rng = random.Random(9200 + seed)
    layers = []
    for _ in range(rng.randint(1, 4)):
        kv_heads, dim = rng.choice([1, 2, 3, 4]), rng.choice([4, 8, 12, 16, 20, 32, 64, 128])
        layers.append(layer(heads=kv_heads * rng.choice([1, 2, 3, 4]), kv_heads=kv_heads, dim=dim, chunk=rng.choice([0, 1, 2, 8, 13, 16, 41, 64]),
                            rot_dims=rng.choice([0, 2, dim // 4 * 2, dim]), base=rng.choice([50.0, 1.0e4, 1.0e6]), scaling=_bands(rng, [10, 40, 200]),
                            scale=rng.uniform(0.5, 1.5) * dim ** -0.5, ff=rng.choice([None, 5, 16, 33, 120])))
    return make_config(layers, width=rng.choice([20, 32, 44, 64, 72, 96]), vocab=rng.randint(50, 200), eps=rng.choice([1e-6, 1e-5]),
                       embedding_scale=rng.choice([0.5, 1.0, 3.0]), residual_mult=rng.choice([0.3, 0.8, 1.0]), loop=_loop(rng, len(layers)))


def test_the_draws_differ():
    drawn = [draw_config(seed) for seed in range(DRAWS)]
    layers = [each for config in drawn for each in config["layers"]]
    assert any("loop" not in config for config in drawn) and any(config.get("loop", {}).get("times", 1) > 1 for config in drawn)
    assert any(each["mlp"] is None for each in layers) and any(each["mlp"] for each in layers)
    assert any("mask" not in each["mixer"] for each in layers) and any("rot" not in each["mixer"] for each in layers)
    assert any((each["mixer"].get("rot") or {}).get("scaling") for each in layers)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("seed", range(DRAWS))
def test_a_drawn_configuration_in_mixed_batches(seed, dtype, tmp_path):
    config = draw_config(seed)
    weights = make_weights(config, seed=100 + seed)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    sequences = _sequences(config, [33, 70, 12, 58, 91, 6], seed=seed)
    double = as_double(weights)
    plain = {rid: forward(config, double, tokens) for rid, tokens in sequences.items()}
    records, peak = mixed(sequences, seed=seed, max_live=3, page=8)
    runner = _runner(folder, config, dtype, peak, page=8, slots=3)
    _compare(_replay(runner, records), plain, dtype, f"seed {seed} {dtype}: {config}")


def draw_large_config(seed: int) -> dict:
    """Sizes nearer to a real model's: widths of a few hundred, heads of 32 to 128, chunks of tens to hundreds."""
    rng = random.Random(640 + seed)
    layers = []
    for _ in range(rng.randint(3, 5)):
        kv_heads, dim = rng.choice([1, 2, 4]), rng.choice([32, 80, 96, 128])
        layers.append(layer(heads=kv_heads * rng.choice([1, 2, 4]), kv_heads=kv_heads, dim=dim, chunk=rng.choice([0, 50, 100, 177, 256]),
                            rot_dims=rng.choice([dim // 2, dim]), base=rng.choice([1e4, 2.5e5]), scaling=_bands(rng, [64, 300]),
                            scale=rng.uniform(0.7, 1.3) * dim ** -0.5, ff=rng.choice([None, 200, 333, 640])))
    return make_config(layers, width=rng.choice([128, 192, 320]), vocab=rng.randint(300, 900), eps=1e-6,
                       embedding_scale=rng.choice([1.0, 12.0]), residual_mult=rng.choice([0.35, 0.8]), loop=_loop(rng, len(layers)))


@pytest.mark.gpu
@pytest.mark.parametrize("seed", range(3))
def test_a_larger_drawn_model_over_hundreds_of_tokens(seed, tmp_path):
    """Float32, a 700-token request whole, with its tail decoded, in portions of changing size, and mixed with shorter
    requests on four slots: every row within 5e-5 of the logits' spread (difference with its mean removed, root mean
    square over the vocabulary), which a key lost far back, a chunk off by one or a pass that read another's cache would
    exceed a thousandfold."""
    config = draw_large_config(seed)
    weights = make_weights(config, seed=500 + seed)
    folder = write_folder(tmp_path / "model", config, weights, torch.float32)
    sequences = _sequences(config, [700, 260, 90, 33, 1], seed=seed)
    double = as_double(weights)
    plain = {rid: forward(config, double, tokens) for rid, tokens in sequences.items()}
    records, peak = mixed(sequences, seed=seed, max_live=4, page=16)
    runner = _runner(folder, config, "float32", max(peak, 704), page=16, slots=4)
    first = sequences["r0"]
    for label, trace in (("whole", whole("r0", first)), ("tail", tail_one_by_one("r0", first, tail=70)),
                         ("portions", portions("r0", first, [37, 37, 14, 19, 6, 2, 128, 1, 1, 64])), ("mixed", records)):
        for rid, by_position in _replay(runner, trace).items():
            positions = sorted(by_position)
            got = torch.stack([by_position[p] for p in positions]).double()
            want = plain[rid][positions]
            error = got - want
            share = (error - error.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.std()
            assert float(share.max()) < 5e-5, f"seed {seed} ({label}): request {rid!r}, position {positions[int(share.argmax())]}: {float(share.max()):.2e}"
