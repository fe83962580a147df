"""The Danalorn decoder in the engine against the plain implementation (``plain_danalorn.py``).

Every configuration of ``danalorn_models.CONFIGS`` runs whole, with its tail decoded token by token, in portions of changing
size down to two tokens, and mixed with other requests on pages and slots that are used again; then the edges: a far key that
stands out among hundreds (before, on and behind a page's border) in both attentions, the keys just inside and just outside a
window, also in layers that read another layer's rows through a narrower and a wider window than its own, windows that let a
small pool serve a long sequence, sinks that take the row, a far token under decays of nearly one, the first tokens of a
sequence on slots used again, the token before across steps, temperatures whose steps fall into portions, long decoding from
captured graphs, long prompts beside each other on the tcgen05 tiles, cached rows wider than the tiles take, greedy
generation through ``LLM.generate``, the command line and the trace runner.
"""

from __future__ import annotations

import dataclasses

import pytest
import torch
from danalorn_models import CONFIGS, as_double, attention_layer, dense, gla_layer, latent_layer, make_config, make_weights, write_folder
from plain_danalorn import forward, greedy
from test_kopatar_gpu import DTYPES, _compare, _replay, _runner, _sequences
from tolerances import assert_rows_close_by_size
from trace_tools import mixed, portions, tail_one_by_one, whole

pytestmark = pytest.mark.gpu


def _plain(sequences, weights, config):
    double = as_double(weights)
    return {rid: forward(tokens, double, config) for rid, tokens in sequences.items()}


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
@pytest.mark.parametrize("name", ["stack", "narrow", "wide heads", "shared rows"])
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
def pointing(config, seed, gain=1.0):
    """Weights of a model whose layers point: token 0's query is token 1's key and no other token's.  Every row of the table
    has mean zero and variance one and token 1's row is token 0's moved one place on; a query's projection is the key's with
    its columns moved one place back.  Token-pair rows, biases and what a position does to a score are small."""
    weights = make_weights(config, seed=seed)
    rows = weights["embed"]
    rows = (rows - rows.mean(-1, keepdim=True)) / rows.std(-1, unbiased=False, keepdim=True)
    rows[1] = torch.roll(rows[0], 1)
    weights["embed"] = rows.bfloat16().float()
    weights["bigram"] = (0.02 * weights["bigram"]).bfloat16().float()
    for index, layer in enumerate(config["layers"]):
        p, sizes = f"l{index}.", layer["mixer"]
        heads, dim = sizes["heads"], sizes["dim"]
        weights[p + "norm1"] = torch.ones_like(weights[p + "norm1"])
        if layer["type"] == "attention":
            keys = torch.roll(weights[p + "mix.k"], -1, dims=1).view(sizes["kv_heads"], dim, -1)
            weights[p + "mix.q"] = keys.repeat_interleave(heads // sizes["kv_heads"], dim=0).reshape(heads * dim, -1).clone()
            for name in ("q", "k"):
                weights[p + f"mix.{name}.b"] = 0 * weights[p + f"mix.{name}.b"]
                weights[p + f"mix.{name}.norm"] = torch.ones(dim)
            continue
        owner = sizes.get("kv_from", index)
        rank, rot = sizes["kv_rank"], sizes["rot_dim"]
        assert sizes["q_rank"] == rank
        weights[p + "mix.dq"] = torch.roll(weights[f"l{owner}.mix.dkv"][:rank], -1, dims=1)
        weights[p + "mix.dq.norm"] = weights[f"l{owner}.mix.dkv.norm"].clone()
        uq = torch.zeros(heads, dim + rot, rank)
        uq[:, :dim] = gain * weights[p + "mix.uk"].view(heads, dim, rank)
        weights[p + "mix.uq"] = uq.view(heads * (dim + rot), rank).bfloat16().float()
    return weights


def _moves(runner, schedules, base, other, last, want, effect, dtype):
    for records_of in schedules:
        got = [_replay(runner, records_of(tokens))["a"][last] for tokens in (base, other)]
        error = float(((got[0] - got[1]) - (want[0] - want[1])).abs().max())
        assert error < (2e-3 if dtype == "float32" else 0.15) * effect


POINTED = {
    "latent": lambda: latent_layer(heads=2, dim=32, rot_dim=8, vdim=24, kv_rank=32, q_rank=32, window=0, scale=0.25),
    "latent, window": lambda: latent_layer(heads=2, dim=32, rot_dim=8, vdim=24, kv_rank=32, q_rank=32, window=399, scale=0.25),
    "attention 32": lambda: attention_layer(heads=8, kv_heads=2, dim=32, vdim=32, scale=1.0, temp=(0.3, 100)),
    "attention 128": lambda: attention_layer(heads=8, kv_heads=4, dim=128, vdim=128, scale=0.25, temp=(0.3, 100)),
}


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("far", [2, 15, 16, 33])
@pytest.mark.parametrize("kind", list(POINTED))
def test_a_far_key_stands_out_among_hundreds(kind, far, dtype, tmp_path):
    """The last token is token 0 and its query points at token 1's key, which stands at one far place among 400
    (before, on and behind a border of the 16-token pages).  Replacing that far token must change the last logits as
    the plain implementation says: in a whole prompt, with the tail decoded, and in portions."""
    config = make_config([POINTED[kind]()], width=32, vocab=40, scale=1.0)
    weights = pointing(config, seed=31)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    generator = torch.Generator().manual_seed(far)
    base = torch.randint(2, config["vocab"], (400,), generator=generator).tolist()
    base[far], base[-1] = 1, 0                      # tokens 0 and 1 nowhere else
    other = list(base)
    other[far] = 2
    last = len(base) - 1
    want = [forward(tokens, as_double(weights), config)[last].float() for tokens in (base, other)]
    effect = float((want[0] - want[1]).abs().max())
    assert effect > 0.2, f"the test's weights do not make the far key count: {effect}"
    runner = _runner(folder, config, dtype, 416, page=16)
    _moves(runner, (lambda t: whole("a", t), lambda t: tail_one_by_one("a", t, tail=20), lambda t: portions("a", t, [150, 2, 99, 17])),
           base, other, last, want, effect, dtype)


WINDOW = 21


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("length", [WINDOW + 1, 112, 129, 140])
@pytest.mark.parametrize("reader", [None, WINDOW - 8, WINDOW + 11, 0])
def test_the_keys_just_inside_and_just_outside_a_window(reader, length, dtype, tmp_path):
    """The last token is token 0, whose query points at token 1's key, which stands at one place: the oldest one the window
    holds must change the last logits as the plain implementation says, the one before it must change nothing; in a whole
    prompt, with the tail decoded until the window has passed over it, and in portions.  With a ``reader`` the window is that
    of a second layer that reads the first one's rows (narrower, wider, all keys), whose own output is switched off."""
    sizes = dict(heads=2, dim=32, rot_dim=8, vdim=24, kv_rank=32, q_rank=32, scale=0.25)
    layers = [latent_layer(window=WINDOW, **sizes)]
    if reader is not None:
        layers.append(latent_layer(window=reader, kv_from=0, **sizes))
    config = make_config(layers, width=32, vocab=40, scale=1.0, buckets=1)
    weights = pointing(config, seed=37)
    # (a single pair row, so that a changed token is felt at its own place alone)
    weights["bigram"] = 0 * weights["bigram"]
    if reader is not None:
        weights["l0.norm1b"] = 0 * weights["l0.norm1b"]
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    double = as_double(weights)
    window = WINDOW if reader is None else reader
    last = length - 1
    runner = _runner(folder, config, dtype, 160, page=16)
    schedules = (lambda t: whole("a", t), lambda t: tail_one_by_one("a", t, tail=window + 6), lambda t: tail_one_by_one("a", t, tail=2),
                 lambda t: portions("a", t, [40, 2, 61, 7, 3]))
    places = [(last - window + 1, True), (last - window, False)] if window else [(0, True), (last // 2, True)]
    for place, inside in places:
        if place < 0:
            continue
        generator = torch.Generator().manual_seed(5)
        base = torch.randint(2, config["vocab"], (length,), generator=generator).tolist()
        base[place], base[-1] = 1, 0
        other = list(base)
        other[place] = 2
        want = [forward(tokens, double, config)[last].float() for tokens in (base, other)]
        effect = float((want[0] - want[1]).abs().max())
        assert (effect > 0.1) == inside, "the plain implementation's window is off by one, or the weights do not point"
        if inside:
            _moves(runner, schedules, base, other, last, want, effect, dtype)
            continue
        for records_of in schedules:
            got = [_replay(runner, records_of(tokens))["a"][last] for tokens in (base, other)]
            assert float((got[0] - got[1]).abs().max()) == 0.0, "a key outside the window reached the logits"


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_windows_give_pages_back_while_a_sequence_grows(dtype, tmp_path):
    """Windowed layers, one of which another layer reads through a wider window, beside recurrent ones: a sequence several
    times longer than the pool runs, in portions and while decoding, because passed pages are handed out again."""
    from rapid_llm_b200.config import load_config
    from rapid_llm_b200.engine.runner import ModelRunner
    from rapid_llm_b200.replay import engine_config_for

    config = make_config([latent_layer(window=9, mlp=dense(24)), gla_layer(), latent_layer(window=20, kv_from=0), latent_layer(window=4, kv_rank=24)], width=48)
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
    _compare(rows, plain, dtype, f"windows on a small pool {dtype}")
    assert len(rows["a"]) == len(tokens)


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_sinks_take_part_of_every_row(dtype, tmp_path):
    """Sinks from far below to far above the scores, one a head: the last kind leaves next to nothing of the values, and a
    token that sees itself alone still shares its row with the sink."""
    config = make_config([latent_layer(heads=4, window=30, scale=0.3)], width=32, vocab=40)
    weights = make_weights(config, seed=3)
    weights["l0.mix.sink"] = torch.tensor([-30.0, 0.0, 4.0, 40.0])
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    tokens = _sequences(config, [70], seed=2)["r0"]
    plain = _plain({"a": tokens}, weights, config)
    runner = _runner(folder, config, dtype, 80, page=16)
    for records in (whole("a", tokens), tail_one_by_one("a", tokens, tail=50), portions("a", tokens, [2, 29, 7])):
        _compare(_replay(runner, records), plain, dtype, f"sinks {dtype}")


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_a_far_token_under_a_decay_of_nearly_one(dtype, tmp_path):
    """With decays of about 0.9995 the first token still weighs at position 300: what changing it does to the last
    logits must match the plain implementation (a state that was lost or restarted on the way would show here)."""
    config = make_config([gla_layer(heads=2, dim=16, vdim=16, tau=4.0, rank=4)], width=32, vocab=50, buckets=1)
    weights = make_weights(config, seed=9)
    weights["bigram"] = 0 * weights["bigram"]
    weights["l0.mix.a2.b"] = torch.full_like(weights["l0.mix.a2.b"], 6.0)
    weights["l0.mix.a2"] = 0 * weights["l0.mix.a2"]
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    generator = torch.Generator().manual_seed(6)
    base = torch.randint(0, config["vocab"], (300,), generator=generator).tolist()
    other = [(base[0] + 7) % config["vocab"]] + base[1:]
    runner = _runner(folder, config, dtype, 320, page=16)
    last = len(base) - 1
    want = [forward(tokens, as_double(weights), config)[last].float() for tokens in (base, other)]
    effect = float((want[0] - want[1]).abs().max())
    assert effect > 5e-3, "the test's weights do not make the far token count"
    for records_of in (lambda t: whole("a", t), lambda t: portions("a", t, [64, 2, 31, 1, 90]), lambda t: tail_one_by_one("a", t, tail=100)):
        got = [_replay(runner, records_of(tokens))["a"][last] for tokens in (base, other)]
        error = float(((got[0] - got[1]) - (want[0] - want[1])).abs().max())
        assert error < (1e-2 * effect if dtype == "float32" else 0.25 * effect + 0.05)


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_the_first_tokens_of_a_sequence(dtype, tmp_path):
    """Positions 0 to 5 alone: the first token takes the pair table's last row, whatever the slot kept from its last owner;
    a window of one position; temperatures that step at every position.  Every slot is used several times."""
    config = make_config([gla_layer(heads=2, mlp=dense(16)), latent_layer(window=1), attention_layer(temp=(0.8, 1)), latent_layer(window=2, kv_from=1)], width=48, buckets=7)
    weights = make_weights(config, seed=41)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    sequences = _sequences(config, [6, 1, 3, 2, 5, 4, 1, 2], seed=9)
    plain = _plain(sequences, weights, config)
    runner = _runner(folder, config, dtype, 32, page=8, slots=2)
    for rid, tokens in sequences.items():
        _compare(_replay(runner, portions(rid, tokens, [1, 2])), plain, dtype, f"first tokens {dtype}")
    records, peak = mixed(sequences, seed=4, max_live=2, page=8)
    _compare(_replay(_runner(folder, config, dtype, peak, page=8, slots=2), records), plain, dtype, f"first tokens {dtype} (mixed)")


def test_the_token_before_belongs_to_the_request(tmp_path):
    """Two requests fed in alternating steps, and a third that takes over a freed slot: the token-pair row and the state
    follow each request, not the batch or the slot."""
    config = make_config([gla_layer(heads=1)], width=24, vocab=30, buckets=29, mul_prev=13, mul_cur=1)
    weights = make_weights(config, seed=43)
    folder = write_folder(tmp_path / "model", config, weights, torch.float32)
    sequences = _sequences(config, [9, 8, 7], seed=1)
    plain = _plain(sequences, weights, config)
    a, b, c = (sequences[r] for r in ("r0", "r1", "r2"))

    def entry(rid, tokens):
        return {"id": rid, "tokens": tokens, "want": list(range(len(tokens)))}

    records = [
        {"step": 0, "entries": [entry("r0", a[:3])], "end": []},
        {"step": 1, "entries": [entry("r1", b[:2])], "end": []},
        {"step": 2, "entries": [entry("r1", b[2:3]), entry("r0", a[3:4])], "end": []},
        {"step": 3, "entries": [entry("r0", a[4:])], "end": ["r0"]},
        {"step": 4, "entries": [entry("r2", c[:1]), entry("r1", b[3:5])], "end": []},
        {"step": 5, "entries": [entry("r1", b[5:]), entry("r2", c[1:])], "end": ["r1", "r2"]},
    ]
    _compare(_replay(_runner(folder, config, "float32", 32, page=8, slots=2), records), plain, "float32", "the token before")


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_long_prompts_on_wide_and_many_heads(dtype, tmp_path):
    """Heads of 128 with and without sharing key heads, heads of 256 and of an odd size, cached rows of 256 with sixteen
    heads; prompts of hundreds of tokens (the library's products), portions behind cached keys, single tokens beside
    portions whose key ranges are split."""
    config = make_config([
        attention_layer(heads=8, kv_heads=2, dim=128, vdim=128, scale=0.1, temp=(0.4, 64), mlp=dense(256)),
        latent_layer(heads=16, dim=24, rot_dim=64, vdim=40, kv_rank=192, q_rank=48, base=1.0e4, window=130, scale=0.12),
        attention_layer(heads=3, kv_heads=3, dim=100, vdim=120, scale=0.1, temp=(0.4, 150), mlp=dense(64)),
        latent_layer(heads=5, dim=40, rot_dim=64, vdim=16, kv_rank=192, q_rank=100, base=1.0e4, window=0, kv_from=1, scale=0.1),
        attention_layer(heads=2, kv_heads=1, dim=256, vdim=200, scale=0.06, temp=None),
        gla_layer(heads=4, dim=64, vdim=128, tau=16.0, rank=16, mlp=dense(200)),
    ], width=128, vocab=150)
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
def test_cached_rows_wider_than_the_tiles_take(dtype, tmp_path):
    """A latent of 300 numbers runs the one-warp-per-row attention in both precisions, window, sink and readers included."""
    config = make_config([latent_layer(heads=3, dim=20, rot_dim=16, vdim=24, kv_rank=300, q_rank=40, window=50, scale=0.1, mlp=dense(48)),
                          latent_layer(heads=2, dim=16, rot_dim=16, vdim=30, kv_rank=300, q_rank=33, window=70, scale=0.1, kv_from=0)], width=64)
    weights = make_weights(config, seed=21)
    folder = write_folder(tmp_path / "model", config, weights, DTYPES[dtype])
    sequences = _sequences(config, [150, 33, 80], seed=5)
    plain = _plain(sequences, weights, config)
    runner = _runner(folder, config, dtype, 160, page=16)
    _compare(_replay(runner, tail_one_by_one("r0", sequences["r0"], tail=80)), plain, dtype, f"wide rows {dtype}")
    records, peak = mixed(sequences, seed=3, max_live=3, page=16)
    _compare(_replay(_runner(folder, config, dtype, peak, page=16, slots=3), records), plain, dtype, f"wide rows {dtype} (mixed)")


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


def test_hundreds_of_keys_decoded_from_captured_graphs(tmp_path):
    """Contexts of several blocks of 128 keys at heads of 128: the tcgen05 decode tiles' key ranges become more as a request
    grows, and every range's slopes count from the query."""
    from rapid_llm_b200.engine.runner import StepEntry

    config = make_config([attention_layer(heads=4, kv_heads=1, dim=128, vdim=128, scale=0.2, temp=(0.5, 256), mlp=dense(64))], width=64, vocab=90)
    weights = make_weights(config, seed=15)
    folder = write_folder(tmp_path / "model", config, weights, torch.bfloat16)
    sequences = _sequences(config, [1300, 610], seed=12)
    plain = _plain(sequences, weights, config)
    runner = _runner(folder, config, "bfloat16", 2 * 1312, page=16, slots=2, graphs=True)
    fed = {"r0": 1200, "r1": 500}
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
    _compare(rows, plain, "bfloat16", "hundreds of keys")


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
        assert output.outputs[0].token_ids == greedy(prompt, as_double(weights), config, 12)


def test_the_command_line_and_the_trace_runner_take_a_danalorn_folder(tmp_path):
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
    assert [int(t) for t in lines[0].split()] == greedy([5, 9, 12, 80, 3], as_double(weights), config, 6)

    tokens = _sequences(config, [30], seed=2)["r0"]
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": tokens[:17], "want": [16]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": tokens[17:], "want": [0, 12]}], "end": ["x"]}]
    out = tmp_path / "out"
    done = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                           "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), cwd=tmp_path,
                          capture_output=True, text=True)
    assert done.returncode == 0, done.stderr
    assert [line for line in done.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1"]
    plain = forward(tokens, as_double(weights), config).float()
    got = torch.from_numpy(np.fromfile(out / "1.f32", dtype="<f4").reshape(2, -1).copy())
    assert_rows_close_by_size(got, plain[[17, 29]], "float32")
