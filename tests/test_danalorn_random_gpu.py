"""Danalorn configurations drawn by seed against the plain implementation: layer orders, head counts and sizes, latents and
their ranks, windows from one position to none, readers of earlier rows, temperatures, decay ranks and taus, feed-forward
sizes and none, the pair table's constants.  Each draw replays a mixed trace (portions of prompts beside decoded tokens on few
pages and three slots) in float32 and bfloat16.

Some draws have feed-forwards of a dozen entries and heads of a few, and rows whose direction 16-bit rounding alone decides:
in bfloat16 a row is held to four times what rounding does to it in the plain implementation (``plain_danalorn.rounding``)
where that is more than the bound of every other row."""

from __future__ import annotations

import random

import pytest
import torch
from danalorn_models import as_double, attention_layer, gla_layer, latent_layer, make_config, make_weights, write_folder
from plain_danalorn import forward, rounding
from test_kopatar_gpu import DTYPES, _compare, _replay, _runner, _sequences
from tolerances import BF16_ROW_RMS
from trace_tools import mixed, portions, tail_one_by_one, whole

DRAWS = 10
STEADY = BF16_ROW_RMS / 4      # rows that rounding moves by more are held to four times that instead


def _mlp(rng, sizes):
    ff = rng.choice(sizes)
    return None if ff is None else {"kind": "dense", "ff": ff}


def _latent(rng, layers, sizes, windows, mlps):
    """A latent layer with rows of its own or, sometimes, one that reads an earlier layer's."""
    owners = [index for index, each in enumerate(layers) if each["type"] == "latent_attention" and "kv_from" not in each["mixer"]]
    dim = rng.choice(sizes["dim"])
    chosen = dict(heads=rng.choice(sizes["heads"]), dim=dim, vdim=rng.choice(sizes["dim"]), q_rank=rng.choice(sizes["rank"]), window=rng.choice(windows),
                  scale=rng.uniform(0.7, 1.5) * dim ** -0.5, mlp=_mlp(rng, mlps))
    if owners and rng.random() < 0.6:
        owner = rng.choice(owners)
        theirs = layers[owner]["mixer"]
        return latent_layer(kv_from=owner, kv_rank=theirs["kv_rank"], rot_dim=theirs["rot_dim"], base=theirs["rot"]["base"], **chosen)
    return latent_layer(kv_rank=rng.choice(sizes["rank"]), rot_dim=rng.choice(sizes["rot"]), base=rng.choice([50.0, 1.0e4, 1.0e6]), **chosen)


def _attention(rng, dims, kv, mlps, strides):
    kv_heads, dim = rng.choice(kv), rng.choice(dims)
    return attention_layer(heads=kv_heads * rng.choice([1, 2, 3]), kv_heads=kv_heads, dim=dim, vdim=rng.choice([dim, rng.choice(dims)]),
                           scale=rng.uniform(0.7, 1.5) * dim ** -0.5, temp=rng.choice([None, (rng.uniform(0.2, 1.0), rng.choice(strides))]), mlp=_mlp(rng, mlps))


def draw_config(seed: int) -> dict:
    rng = random.Random(7100 + seed)
    layers = []
    for _ in range(rng.randint(2, 5)):
        kind, mlps = rng.choice(["latent", "latent", "attention", "gla"]), [None, 12, 16, 33, 120]
        if kind == "latent":
            layers.append(_latent(rng, layers, {"dim": [4, 7, 16, 20], "heads": [1, 2, 3, 5, 8], "rank": [6, 13, 24, 40], "rot": [2, 6, 8, 16]},
                                  [0, 1, 2, 8, 13, 16, 41], mlps))
        elif kind == "attention":
            layers.append(_attention(rng, [4, 8, 10, 16, 20, 32, 64, 128], [1, 2, 3, 4], mlps, [1, 7, 16, 40]))
        else:
            layers.append(gla_layer(heads=rng.choice([1, 2, 3, 5]), dim=rng.choice([3, 8, 16, 30]), vdim=rng.choice([4, 9, 16, 32]),
                                    tau=rng.choice([1.0, 3.0, 16.0]), rank=rng.choice([1, 4, 7, 16, 33]), mlp=_mlp(rng, mlps)))
    return make_config(layers, width=rng.choice([20, 32, 44, 64, 72, 96]), vocab=rng.randint(50, 200), eps=rng.choice([1e-6, 1e-5]),
                       scale=rng.choice([0.5, 1.0, 6.0]), buckets=rng.choice([1, 17, 251]), mul_prev=rng.choice([1, 37]), mul_cur=rng.choice([1, 5]))


def test_the_draws_differ():
    drawn = [draw_config(seed) for seed in range(DRAWS)]
    layers = [each for config in drawn for each in config["layers"]]
    assert {each["type"] for each in layers} == {"latent_attention", "attention", "gla"}
    assert any("kv_from" in each["mixer"] for each in layers) and any(each["mlp"] is None for each in layers) and any(each["mlp"] for each in layers)
    latents = [each["mixer"] for each in layers if each["type"] == "latent_attention"]
    assert any("mask" not in each for each in latents) and any("mask" in each for each in latents)
    soft = [each["mixer"] for each in layers if each["type"] == "attention"]
    assert any(each["heads"] > each["kv_heads"] for each in soft) and any("q_temp" not in each for each in soft)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("seed", range(DRAWS))
def test_a_drawn_configuration_in_mixed_batches(seed, dtype, tmp_path):
    config = draw_config(seed)
    weights = make_weights(config, seed=100 + seed)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    sequences = _sequences(config, [33, 70, 12, 58, 91, 6], seed=seed)
    double = as_double(weights)
    plain = {rid: forward(tokens, double, config) for rid, tokens in sequences.items()}
    records, peak = mixed(sequences, seed=seed, max_live=3, page=8)
    runner = _runner(folder, config, dtype, peak, page=8, slots=3)
    rows = _replay(runner, records)
    if dtype == "bfloat16":
        for rid, tokens in sequences.items():
            moved = rounding(tokens, double, config, torch.bfloat16, plain[rid])
            for position in [at for at in rows.get(rid, {}) if float(moved[at]) > STEADY]:
                got, want = rows[rid].pop(position).double(), plain[rid][position]
                error, size = got - want, (want - want.mean()).square().mean().sqrt()
                share = float((error - error.mean()).square().mean().sqrt() / size)
                assert share <= 4 * float(moved[position]), f"seed {seed}: request {rid!r}, position {position}: {share:.4f}, rounding moves {float(moved[position]):.4f}"
        rows = {rid: by_position for rid, by_position in rows.items() if by_position}
    _compare(rows, plain, dtype, f"seed {seed} {dtype}: {config}")


def draw_large_config(seed: int) -> dict:
    """Sizes nearer to a real model's: widths of a few hundred, heads of 32 to 128, windows of tens to hundreds."""
    rng = random.Random(820 + seed)
    layers = []
    for place in range(rng.randint(4, 6)):
        kind, mlps = ["latent", "attention", "gla"][(place + seed) % 3], [None, 200, 333, 640]
        if kind == "latent" or rng.random() < 0.2:
            layers.append(_latent(rng, layers, {"dim": [32, 48, 64], "heads": [2, 4, 7], "rank": [64, 100, 160], "rot": [16, 32, 64]},
                                  [0, 50, 100, 177, 256], mlps))
        elif kind == "attention":
            layers.append(_attention(rng, [32, 80, 96, 128], [1, 2, 4], mlps, [50, 128, 300]))
        else:
            layers.append(gla_layer(heads=rng.choice([2, 4, 6]), dim=rng.choice([32, 48, 64]), vdim=rng.choice([32, 64, 80]),
                                    tau=rng.choice([8.0, 16.0]), rank=rng.choice([16, 24]), mlp=_mlp(rng, mlps)))
    return make_config(layers, width=rng.choice([128, 192, 320]), vocab=rng.randint(300, 900), eps=1e-6,
                       scale=rng.choice([1.0, 9.0]), buckets=rng.choice([509, 2003]), mul_prev=rng.choice([31, 211]), mul_cur=rng.choice([3, 11]))


@pytest.mark.gpu
@pytest.mark.parametrize("seed", range(3))
def test_a_larger_drawn_model_over_hundreds_of_tokens(seed, tmp_path):
    """Float32, a 700-token request whole, with its tail decoded, in portions of changing size, and mixed with shorter
    requests on four slots: every row within 5e-5 of the logits' spread (difference with its mean removed, root mean
    square over the vocabulary), which a key lost far back, a window off by one or a state that was lost would exceed a
    thousandfold."""
    config = draw_large_config(seed)
    weights = make_weights(config, seed=500 + seed)
    folder = write_folder(tmp_path / "model", config, weights, torch.float32)
    sequences = _sequences(config, [700, 260, 90, 33, 1], seed=seed)
    double = as_double(weights)
    plain = {rid: forward(tokens, double, config) for rid, tokens in sequences.items()}
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
