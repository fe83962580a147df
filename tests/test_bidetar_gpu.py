"""The Bidetar decoder in the engine against the plain implementation (``plain_bidetar.py``).

Every configuration of ``bidetar_models.CONFIGS`` runs whole, with its tail decoded token by token, in portions of
changing size down to two tokens, and mixed with other requests on pages and slots that are used again; then the edges:
a far key that stands out among hundreds (before, on and behind a page's border), the keys just inside and just outside a
chunk in prompts and while decoding, chunks that let a small pool serve a long sequence, a sink that takes the row, the
first tokens of a sequence on slots used again, long decoding from captured graphs across many chunks, long prompts
beside each other on the tcgen05 tiles, the sublayers' products unstacked, greedy generation through ``LLM.generate``,
the command line and the trace runner.
"""

from __future__ import annotations

import dataclasses

import pytest
import torch
from bidetar_models import BANDS, CONFIGS, as_double, layer, make_config, make_weights, write_folder
from plain_bidetar import forward, greedy
from test_kopatar_gpu import DTYPES, _compare, _replay, _runner, _sequences
from tolerances import assert_rows_close_by_size
from trace_tools import mixed, portions, tail_one_by_one, whole

pytestmark = pytest.mark.gpu


def _plain(sequences, weights, config):
    double = as_double(weights)
    return {rid: forward(config, double, tokens) for rid, tokens in sequences.items()}


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_decoded_and_in_portions(name, dtype, tmp_path):
    config = CONFIGS[name]
    weights = make_weights(config, seed=11)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    tokens = _sequences(config, [93], seed=3)["r0"]
    plain = _plain({"a": tokens}, weights, config)
    runner = _runner(folder, config, dtype, 160)
    for label, records in (
        ("whole", whole("a", tokens)),
        ("tail one by one", tail_one_by_one("a", tokens, tail=50)),
        ("portions", portions("a", tokens, [2, 3, 16, 2, 7, 8, 1, 5])),
        ("portions of two", portions("a", tokens, [2])),
        ("token by token", portions("a", tokens, [1])),
    ):
        _compare(_replay(runner, records), plain, dtype, f"{name} {dtype} ({label})")


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("name", ["stack", "narrow", "wide heads"])
def test_mixed_batches_on_reused_pages_and_slots(name, dtype, tmp_path):
    config = CONFIGS[name]
    weights = make_weights(config, seed=5)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    sequences = _sequences(config, [37, 90, 18, 75, 131, 52, 9], seed=8)
    plain = _plain(sequences, weights, config)
    records, peak = mixed(sequences, seed=2, max_live=3, page=8)
    runner = _runner(folder, config, dtype, peak, page=8, slots=3)
    mixed_rows = _replay(runner, records)
    _compare(mixed_rows, plain, dtype, f"{name} {dtype} (mixed)")
    # the same requests alone: what else is in the batch, and which slot and pages serve, changes nothing but rounding
    if dtype == "float32":
        for rid in ("r1", "r4"):
            alone = _replay(runner, whole(rid, sequences[rid]))[rid]
            for position, row in mixed_rows[rid].items():
                torch.testing.assert_close(row, alone[position], rtol=2e-5, atol=2e-5)


# ------------------------------------------------------------------ keys that stand out -- #
def pointing(config, seed, gain=3.0):
    """Weights of a one-layer model in which token 0's query points at token 1's key and at no other: every row of the
    table has mean zero and variance one, so the norm in front of the layer (weight one) hands it on as it is; token 1's
    row is token 0's with its entries moved one place on, and the query projection is the key projection with its columns
    moved one place back, so ``W_q x_0 = W_k x_1``.  The norm weight of k is one, that of q the gain, biases are small, and
    so is the rotated share of a head: positions hardly move a score."""
    weights = make_weights(config, seed=seed)
    rows = weights["embed"]
    rows = (rows - rows.mean(-1, keepdim=True)) / rows.std(-1, unbiased=False, keepdim=True)
    rows[1] = torch.roll(rows[0], 1)
    weights["embed"] = (rows / config["embedding"]["scale"]).bfloat16().float()
    sizes = config["layers"][0]["mixer"]
    heads, dim = sizes["heads"], sizes["dim"]
    keys = torch.roll(weights["l0.mix.k"], -1, dims=1).view(sizes["kv_heads"], dim, -1)
    weights["l0.norm1"] = torch.ones_like(weights["l0.norm1"])
    weights["l0.mix.q"] = keys.repeat_interleave(heads // sizes["kv_heads"], dim=0).reshape(heads * dim, -1).clone()
    for name in ("q", "k"):
        weights[f"l0.mix.{name}.b"] = (0.1 * weights[f"l0.mix.{name}.b"]).bfloat16().float()
    weights["l0.mix.q.norm"] = torch.full_like(weights["l0.mix.q.norm"], gain)
    weights["l0.mix.k.norm"] = torch.ones_like(weights["l0.mix.k.norm"])
    return weights


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("far", [2, 15, 16, 33])
@pytest.mark.parametrize("dim,chunk", [(32, 0), (32, 500), (128, 410)])
def test_a_far_key_stands_out_among_hundreds(dim, chunk, far, dtype, tmp_path):
    """The last token is token 0 and its query points at token 1's key, which stands at one far place among 400
    (before, on and behind a border of the 16-token pages).  Replacing that far token must change the last logits as
    the plain implementation says: in a whole prompt, with the tail decoded, and in portions."""
    config = make_config([layer(heads=4, kv_heads=2, dim=dim, chunk=chunk, rot_dims=4, scale=8.0 / dim, ff=24)], width=32, vocab=40)
    weights = pointing(config, seed=31)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    generator = torch.Generator().manual_seed(far)
    base = torch.randint(2, config["vocab"], (400,), generator=generator).tolist()
    base[far], base[-1] = 1, 0                      # tokens 0 and 1 nowhere else
    other = list(base)
    other[far] = 2
    last = len(base) - 1
    want = [forward(config, as_double(weights), tokens)[last].float() for tokens in (base, other)]
    effect = float((want[0] - want[1]).abs().max())
    assert effect > 0.2, "the test's weights do not make the far key count"
    runner = _runner(folder, config, dtype, 416, page=16)
    for records_of in (lambda t: whole("a", t), lambda t: tail_one_by_one("a", t, tail=20), lambda t: portions("a", t, [150, 2, 99, 17])):
        got = [_replay(runner, records_of(tokens))["a"][last] for tokens in (base, other)]
        error = float(((got[0] - got[1]) - (want[0] - want[1])).abs().max())
        assert error < (2e-3 if dtype == "float32" else 0.15) * effect


CHUNK = 21


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("length", [CHUNK * 6 + 1, CHUNK * 6 + 15, CHUNK * 7])
@pytest.mark.parametrize("dim", [32, 128])
def test_the_keys_just_inside_and_just_outside_a_chunk(dim, length, dtype, tmp_path):
    """A query sees the first position of its own chunk and not the one before it, however near that is.  The last token
    (the first, the fifteenth and the last of its chunk) is token 0, whose query points at token 1's key, which stands at
    one place: at the chunk's start it must change the last logits as the plain implementation says, right before it it
    must change nothing; in a whole prompt, with the tail decoded across the border, and in portions that cut the chunk."""
    config = make_config([layer(heads=2, kv_heads=2, dim=dim, chunk=CHUNK, rot_dims=4, scale=8.0 / dim)], width=32, vocab=40)
    weights = pointing(config, seed=37)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    double = as_double(weights)
    generator = torch.Generator().manual_seed(5)
    last = length - 1
    start = last // CHUNK * CHUNK
    runner = _runner(folder, config, dtype, 160, page=16)
    schedules = (lambda t: whole("a", t), lambda t: tail_one_by_one("a", t, tail=last - start + 4), lambda t: tail_one_by_one("a", t, tail=2),
                 lambda t: portions("a", t, [40, 2, 61, 7, 3]))
    for place, inside in ((start, True), (start - 1, False)):
        if place == last:                          # the query at a chunk's first position sees itself alone
            continue
        base = torch.randint(2, config["vocab"], (length,), generator=generator).tolist()
        base[place], base[-1] = 1, 0
        other = list(base)
        other[place] = 2
        want = [forward(config, double, tokens)[last].float() for tokens in (base, other)]
        effect = float((want[0] - want[1]).abs().max())
        assert (effect > 0.1) == inside, "the plain implementation's chunk is off by one, or the weights do not point"
        for records_of in schedules:
            got = [_replay(runner, records_of(tokens))["a"][last] for tokens in (base, other)]
            moved = got[0] - got[1]
            if inside:
                assert float((moved - (want[0] - want[1])).abs().max()) < (2e-3 if dtype == "float32" else 0.15) * effect
            else:
                assert float(moved.abs().max()) == 0.0, "a key of the chunk before reached the logits"


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_chunks_give_pages_back_while_a_sequence_grows(dtype, tmp_path):
    """A looped model of chunked layers only runs a sequence several times longer than the pool: the pages of passed
    chunks are handed out again, in portions and while decoding, and the logits stay those of the plain implementation."""
    from rapid_llm_b200.config import load_config
    from rapid_llm_b200.engine.runner import ModelRunner
    from rapid_llm_b200.replay import engine_config_for

    config = make_config([layer(chunk=9, ff=32), layer(chunk=14)], width=48, loop=(0, 1, 2))
    weights = make_weights(config, seed=19)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    tokens = _sequences(config, [150], seed=1)["r0"]
    plain = _plain({"a": tokens}, weights, config)
    engine = dataclasses.replace(engine_config_for(load_config(folder), dtype, 160, 8, 2), num_pages=6)    # 48 of 150 tokens
    runner = ModelRunner.from_folder(folder, engine)
    records = portions("a", tokens[:60], [9, 2, 16, 5])
    records[-1]["end"] = []
    for offset, token in enumerate(tokens[60:]):
        records.append({"step": 100 + offset, "entries": [{"id": "a", "tokens": [token], "want": [0]}], "end": []})
    records[-1]["end"] = ["a"]
    rows = _replay(runner, records)
    _compare(rows, plain, dtype, f"chunks on a small pool {dtype}")
    assert len(rows["a"]) == len(tokens)


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("dim", [16, 128])
def test_a_sink_takes_part_of_every_row(dim, dtype, tmp_path):
    """Sinks from far below to far above the scores, one a head: the second kind leaves next to nothing of the values, and
    a token that sees itself alone still shares its row with the sink."""
    config = make_config([layer(heads=4, kv_heads=1, dim=dim, chunk=30, rot_dims=8, scale=0.2)], width=32, vocab=40)
    weights = make_weights(config, seed=3)
    weights["l0.mix.sink"] = torch.tensor([-30.0, 0.0, 4.0, 40.0])
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    tokens = _sequences(config, [70], seed=2)["r0"]
    plain = _plain({"a": tokens}, weights, config)
    runner = _runner(folder, config, dtype, 80, page=16)
    for records in (whole("a", tokens), tail_one_by_one("a", tokens, tail=50), portions("a", tokens, [2, 29, 7])):
        _compare(_replay(runner, records), plain, dtype, f"sinks {dim} {dtype}")


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_the_first_tokens_of_a_sequence(dtype, tmp_path):
    """Positions 0 to 5 alone, chunks of two, three and one positions.  Every slot is used several times."""
    config = make_config([layer(chunk=3, ff=16), layer(chunk=2), layer(chunk=1, ff=8)], width=48, loop=(1, 3, 2))
    weights = make_weights(config, seed=41)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    sequences = _sequences(config, [6, 1, 3, 2, 5, 4, 1, 2], seed=9)
    plain = _plain(sequences, weights, config)
    runner = _runner(folder, config, dtype, 32, page=8, slots=2)
    for rid, tokens in sequences.items():
        _compare(_replay(runner, portions(rid, tokens, [1, 2])), plain, dtype, f"first tokens {dtype}")
    records, peak = mixed(sequences, seed=4, max_live=2, page=8)
    _compare(_replay(_runner(folder, config, dtype, peak, page=8, slots=2), records), plain, dtype, f"first tokens {dtype} (mixed)")


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_long_prompts_on_wide_and_many_heads(dtype, tmp_path):
    """Heads of 128 in chunks of several blocks of keys and without chunks, sixteen heads over one, heads of 256 and of
    an odd size; prompts of hundreds of tokens (the library's products), portions behind cached keys, single tokens beside
    portions whose key ranges are split."""
    config = make_config([
        layer(heads=4, kv_heads=2, dim=128, chunk=150, rot_dims=128, base=1.0e4, scaling=BANDS, scale=0.06, ff=256),
        layer(heads=16, kv_heads=1, dim=24, chunk=128, rot_dims=24, base=1.0e4, scale=0.2),
        layer(heads=4, kv_heads=2, dim=128, chunk=0, rot_dims=64, base=1.0e5, scale=0.06, ff=64),
        layer(heads=2, kv_heads=1, dim=256, chunk=64, rot_dims=128, base=1.0e5, scaling=BANDS, scale=0.04),
    ], width=128, vocab=150, residual_mult=0.5, loop=(0, 2, 2))
    weights = make_weights(config, seed=61)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    sequences = _sequences(config, [400, 45, 290], seed=5)
    plain = _plain(sequences, weights, config)
    runner = _runner(folder, config, dtype, 416, page=16)
    tokens = sequences["r0"]
    _compare(_replay(runner, whole("r0", tokens)), plain, dtype, f"long prompts {dtype} (whole)")
    _compare(_replay(runner, portions("r0", tokens, [130, 2, 90, 1, 40])), plain, dtype, f"long prompts {dtype} (portions)")
    _compare(_replay(runner, tail_one_by_one("r0", tokens, tail=12)), plain, dtype, f"long prompts {dtype} (tail)")
    records, peak = mixed(sequences, seed=3, max_live=3, page=16)
    _compare(_replay(_runner(folder, config, dtype, peak, page=16, slots=3), records), plain, dtype, f"long prompts {dtype} (mixed)")


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("name", ["stack", "wide heads"])
def test_long_decoding_from_captured_graphs(name, dtype, tmp_path):
    from rapid_llm_b200.engine.runner import StepEntry

    config = CONFIGS[name]
    weights = make_weights(config, seed=13)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    sequences = _sequences(config, [150, 171, 160], seed=12)
    plain = _plain(sequences, weights, config)
    runner = _runner(folder, config, dtype, 3 * 176, page=16, slots=4, graphs=True)
    heads = {"r0": 5, "r1": 40, "r2": 2}
    fed = {}
    for rid, head in heads.items():
        assert runner.admit(rid)
        runner.step([StepEntry(rid, sequences[rid][:head], [])])
        fed[rid] = head
    rows = {rid: {} for rid in sequences}
    while any(fed[rid] < len(sequences[rid]) for rid in sequences):
        live = [rid for rid in sequences if fed[rid] < len(sequences[rid])]
        logits = runner.step_decode([StepEntry(rid, [sequences[rid][fed[rid]]], [0]) for rid in live]).float().cpu()
        for row, rid in enumerate(live):
            rows[rid][fed[rid]] = logits[row].clone()
            fed[rid] += 1
    runner.check_fault()
    _compare(rows, plain, dtype, f"long decoding {name} {dtype}")


def test_chunks_of_several_blocks_decoded_from_captured_graphs(tmp_path):
    """Chunks of 600 positions at heads of 128: as a request walks through its chunk the tcgen05 decode tiles' key ranges
    become more and then one again; every step past the prompt is replayed or captured on the way, over two borders."""
    from rapid_llm_b200.engine.runner import StepEntry

    config = make_config([layer(heads=2, kv_heads=1, dim=128, chunk=600, rot_dims=128, base=1.0e4, scaling=BANDS, scale=0.06, ff=64)],
                         width=64, vocab=90)
    weights = make_weights(config, seed=15)
    folder = write_folder(tmp_path / "model", config, weights, torch.bfloat16)
    sequences = _sequences(config, [1300, 610], seed=12)
    double = as_double(weights)
    plain = {rid: forward(config, double, tokens) for rid, tokens in sequences.items()}
    runner = _runner(folder, config, "bfloat16", 2 * 1312, page=16, slots=2, graphs=True)
    fed = {"r0": 1100, "r1": 510}
    for rid, head in fed.items():
        assert runner.admit(rid)
        runner.step([StepEntry(rid, sequences[rid][:head], [])])
    rows = {rid: {} for rid in sequences}
    while any(fed[rid] < len(sequences[rid]) for rid in sequences):
        live = [rid for rid in sequences if fed[rid] < len(sequences[rid])]
        logits = runner.step_decode([StepEntry(rid, [sequences[rid][fed[rid]]], [0]) for rid in live]).float().cpu()
        for row, rid in enumerate(live):
            rows[rid][fed[rid]] = logits[row].clone()
            fed[rid] += 1
    runner.check_fault()
    _compare(rows, plain, "bfloat16", "chunks of several blocks")


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_the_sublayers_products_need_not_be_stacked(dtype, tmp_path, monkeypatch):
    """An arrangement whose sublayers cannot share their products runs each by itself and adds the results: the same
    model with stacking switched off, with and without a feed-forward."""
    from rapid_llm_b200.parts.attention import GQAAttention

    config = CONFIGS["stack"]
    weights = make_weights(config, seed=11)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    sequences = _sequences(config, [60, 90], seed=3)
    plain = _plain(sequences, weights, config)
    monkeypatch.setattr(GQAAttention, "stacks", False)
    runner = _runner(folder, config, dtype, 96, page=8)
    assert not any(block.stacked for block in runner.model.layers)
    _compare(_replay(runner, tail_one_by_one("r0", sequences["r0"], tail=30)), plain, dtype, f"unstacked {dtype}")
    _compare(_replay(runner, portions("r1", sequences["r1"], [70, 2, 5])), plain, dtype, f"unstacked {dtype} (portions)")


def test_greedy_generation_through_the_entry_point(tmp_path):
    """More prompts than slots, so requests wait, and slots and pages change hands; float32 picks the same tokens."""
    from rapid_llm_b200 import LLM, SamplingParams

    config = CONFIGS["stack"]
    weights = make_weights(config, seed=17)
    folder = write_folder(tmp_path / "model", config, weights, torch.float32)
    prompts = list(_sequences(config, [5, 23, 2, 41, 12], seed=14).values())
    llm = LLM(folder, dtype="float32", max_seq_len=96, max_gpu_num_blocks=24, page_size=8, max_num_seqs=2, max_chunk_size=16)
    outputs = llm.generate(prompts, SamplingParams.greedy(max_gen_len=12))
    for prompt, output in zip(prompts, outputs):
        assert output.outputs[0].token_ids == greedy(config, as_double(weights), prompt, 12)


def test_the_command_line_and_the_trace_runner_take_a_bidetar_folder(tmp_path):
    """``batch`` generates from token-id prompts; ``bin/trace_run`` replays steps and writes the same logits as the
    plain implementation computes."""
    import json
    import subprocess
    import sys
    from pathlib import Path

    import numpy as np

    root = Path(__file__).resolve().parents[1]
    config = CONFIGS["stack"]
    weights = make_weights(config, seed=23)
    folder = write_folder(tmp_path / "model", config, weights, torch.float32)
    prompts = tmp_path / "prompts.txt"
    prompts.write_text("5 9 12 80 3\n7 7 1\n")
    done = subprocess.run([sys.executable, "-m", "rapid_llm_b200.cli", "batch", "--model-dir", str(folder), "--dtype", "float32",
                           "--prompt-ids-file", str(prompts), "--max-gen-len", "6", "--temperature", "0", "--repetition-penalty", "1.0", "--max-seq-len", "64",
                           "--max-gpu-num-blocks", "16"], cwd=root, capture_output=True, text=True)
    assert done.returncode == 0, done.stderr
    lines = [line for line in done.stdout.splitlines() if line and not line.startswith("---")]
    assert [int(t) for t in lines[0].split()] == greedy(config, as_double(weights), [5, 9, 12, 80, 3], 6)

    tokens = _sequences(config, [30], seed=2)["r0"]
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": tokens[:17], "want": [16]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": tokens[17:], "want": [0, 12]}], "end": ["x"]}]
    out = tmp_path / "out"
    done = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                           "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), cwd=tmp_path,
                          capture_output=True, text=True)
    assert done.returncode == 0, done.stderr
    assert [line for line in done.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1"]
    plain = forward(config, as_double(weights), tokens).float()
    got = torch.from_numpy(np.fromfile(out / "1.f32", dtype="<f4").reshape(2, -1).copy())
    assert_rows_close_by_size(got, plain[[17, 29]], "float32")
