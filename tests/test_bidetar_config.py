"""Bidetar's configuration on the CPU: parts and their parameters, expected tensors, the run order, where the stacked
weights lie, refusals; chunks in the cache manager and in the planner; the plain implementation against second forms of
the same equations; and that every mechanism of the plain implementation moves the logits of the test models (so a
comparison with it has teeth)."""

from __future__ import annotations

import copy
import math

import numpy as np
import plain_bidetar
import pytest
import torch
from bidetar_models import BANDS, CONFIGS, as_double, layer, make_config, make_weights, tensor_shapes, write_folder
from plain_bidetar import attention_mixer, forward, frequencies, keys_and_values, rms_norm, rotate_neighbours, run_order

from rapid_llm_b200.cache import CacheManager, plan_groups
from rapid_llm_b200.config import BidetarConfig, load_config, resolve_architecture
from rapid_llm_b200.models.causal_lm import CausalLM
from rapid_llm_b200.ops import kernels
from rapid_llm_b200.parts.attention import AttentionItems
from rapid_llm_b200.parts.base import POSITION_ENCODINGS, CacheNeed, StepShape
from rapid_llm_b200.weights import load_weights, write_random_model


def _model(config, dtype=torch.float32):
    return CausalLM(BidetarConfig.from_dict(config).to_spec(), dtype, "cpu")


# ------------------------------------------------------------------------------- configuration -- #
def test_the_registry_finds_the_architecture():
    assert resolve_architecture({"architecture": "Bidetar"}) is BidetarConfig


@pytest.mark.parametrize("name", list(CONFIGS))
def test_the_model_expects_the_files_tensors(name):
    assert {n: tuple(s.shape) for n, s in _model(CONFIGS[name]).tensor_specs().items()} == tensor_shapes(CONFIGS[name])


def test_parts_run_order_and_caches():
    config = CONFIGS["stack"]
    spec = BidetarConfig.from_dict(config).to_spec()
    assert [each.arrangement for each in spec.layers] == ["shared_norm"] * 4
    assert [entry.layer for entry in spec.schedule] == [0, 1, 0, 1, 2, 3] == run_order(4, config["loop"])
    assert all(entry.pass_index is None and entry.cache_from is None for entry in spec.schedule)
    assert [each.mixer.params["chunk"] for each in spec.layers] == [9, 33, 0, 16]
    assert [each.mixer.params["position"].kind for each in spec.layers] == ["rotary_frequencies", "banded_frequencies",
                                                                            "rotary_frequencies", "banded_frequencies"]
    params = spec.layers[1].mixer.params
    assert (params["values_from_keys"], params["qkv_bias"], params["o_bias"], params["sink"], params["gate"], params["rotation"],
            params["qk_norm_over"]) == (True, True, True, True, "sigmoid_head", "neighbours", "row")
    assert spec.layers[1].feed_forward is None and spec.layers[0].feed_forward.params["activation"] == "relu_squared"
    assert spec.layers[0].norm.params["add_scale"] == spec.final_norm.params["add_scale"] == 0.45
    assert spec.embedding.params["scale"] == 0.7 and spec.embedding.params["opens_stream"]
    needs = CausalLM(spec, torch.float32, "cpu").cache_needs()
    assert [(need.kind, need.chunk) for need in needs] == [("chunk", 9), ("chunk", 33), ("chunk", 9), ("chunk", 33), ("full", 0), ("chunk", 16)]
    groups, entry_group = plan_groups(needs)
    assert len(groups) == 4 and entry_group == [0, 1, 0, 1, 2, 3]           # the passes of a layer share page ids, not pages
    # no mask, no rotation, no loop, no constants in the file
    bare = make_config([layer(chunk=0, rot_dims=0)])
    del bare["residual_mult"], bare["embedding"], bare["layers"][0]["mixer"]["vdim"]
    spec = BidetarConfig.from_dict(bare).to_spec()
    assert spec.layers[0].mixer.params["chunk"] == 0 and spec.layers[0].mixer.params["position"].params["rotary_dim"] == 0
    assert spec.layers[0].norm.params["add_scale"] == 1.0 and spec.embedding.params["scale"] == 1.0 and len(spec.schedule) == 1
    assert BidetarConfig.from_dict(BidetarConfig.from_dict(config).to_dict()).to_spec() == BidetarConfig.from_dict(config).to_spec()


@pytest.mark.parametrize("name", ["stack", "narrow"])
def test_where_the_stacked_weights_lie(name, tmp_path):
    """The first product's rows are [up, q, k, gate], the last one's columns [down, o], heads laid out in steps of 16 with
    zeros behind them; loading fills the arrangement's matrices through the parts' views."""
    config = CONFIGS[name]
    weights = make_weights(config, seed=1)
    model = _model(config)
    load_weights(model, write_folder(tmp_path / "model", config, weights, torch.float32))
    for index, (each, block) in enumerate(zip(config["layers"], model.layers)):
        p, m = f"l{index}.", each["mixer"]
        assert block.stacked
        d = -(-m["dim"] // 16) * 16
        ff = 0 if each["mlp"] is None else each["mlp"]["ff"]
        ff8 = -(-ff // 8) * 8
        q, k = m["heads"] * d, m["kv_heads"] * d
        assert block.first.shape == (ff8 + q + k + -(-m["heads"] // 8) * 8, config["width"])
        assert block.last.shape == (config["width"], ff8 + q)
        if ff:
            assert torch.equal(block.first[:ff], weights[p + "mlp.up"]) and torch.equal(block.last[:, :ff], weights[p + "mlp.down"])
        for at, count, name_ in ((ff8, m["heads"], "q"), (ff8 + q, m["kv_heads"], "k")):
            rows = block.first[at : at + count * d].view(count, d, -1)
            assert torch.equal(rows[:, : m["dim"]].reshape(count * m["dim"], -1), weights[p + "mix." + name_])
            assert not rows[:, m["dim"]:].any()
            bias = block.first_bias[at : at + count * d].view(count, d)
            assert torch.equal(bias[:, : m["dim"]].reshape(-1), weights[p + "mix." + name_ + ".b"]) and not bias[:, m["dim"]:].any()
        gate = ff8 + q + k
        assert torch.equal(block.first[gate : gate + m["heads"]], weights[p + "mix.g"]) and not block.first_bias[gate:].any()
        heads = block.last[:, ff8:].view(config["width"], m["heads"], d)
        assert torch.equal(heads[:, :, : m["dim"]].reshape(config["width"], -1), weights[p + "mix.o"]) and not heads[:, :, m["dim"]:].any()
        # everything the zeros do not cover is accounted for
        assert not block.first[ff:ff8].any() and not block.first_bias[:ff8].any() and not block.last[:, ff:ff8].any()


def test_a_random_model_folder_round_trip(tmp_path):
    config = BidetarConfig.from_dict(CONFIGS["loop"])
    folder = write_random_model(tmp_path / "model", config, seed=3, dtype=torch.bfloat16)
    loaded = load_config(folder)
    assert isinstance(loaded, BidetarConfig) and loaded.to_spec() == config.to_spec()
    model = CausalLM(loaded.to_spec(), torch.bfloat16, "cpu")
    counts = load_weights(model, folder)
    assert counts["tensors"] == len(tensor_shapes(CONFIGS["loop"]))
    used = model.parameter_bytes()
    exact = sum((2 if len(shape) == 2 else 4) * math.prod(shape) for shape in tensor_shapes(CONFIGS["loop"]).values())
    assert exact <= used <= 1.05 * exact           # the gates' rows are rounded up to eight, biases cover every row


def test_refusals():
    config = copy.deepcopy(CONFIGS["mixer"])
    config["layers"][0]["type"] = "latent_attention"
    with pytest.raises(ValueError, match="unknown mixer type"):
        BidetarConfig.from_dict(config)
    config = copy.deepcopy(CONFIGS["parallel"])
    config["layers"][0]["mlp"]["kind"] = "moe"
    with pytest.raises(ValueError, match="unknown feed-forward kind"):
        BidetarConfig.from_dict(config)
    config = copy.deepcopy(CONFIGS["mixer"])
    config["layers"][0]["mixer"]["vdim"] = 8
    with pytest.raises(ValueError, match="vdim"):
        BidetarConfig.from_dict(config)
    config = copy.deepcopy(CONFIGS["mixer"])
    del config["layers"][0]["mixer"]["kv_heads"]
    with pytest.raises(ValueError, match="kv_heads"):
        BidetarConfig.from_dict(config)
    config = copy.deepcopy(CONFIGS["parallel"])
    del config["layers"][0]["mixer"]["rot"]["scaling"]["low"]
    with pytest.raises(ValueError, match="low"):
        BidetarConfig.from_dict(config)
    config = copy.deepcopy(CONFIGS["mixer"])
    del config["width"]
    with pytest.raises(ValueError, match="width"):
        BidetarConfig.from_dict(config)
    for loop in ((1, 1, 2), (0, 2, 2), (0, 1, 0)):
        with pytest.raises(ValueError, match="loop"):
            BidetarConfig.from_dict(make_config([layer()], loop=loop))
    # the parts refuse what their kernels do not compute
    from rapid_llm_b200.config.model_spec import PartSpec
    from rapid_llm_b200.parts.base import MIXERS

    base = BidetarConfig.from_dict(CONFIGS["mixer"]).to_spec().layers[0].mixer
    build = lambda **changes: MIXERS.build(base.with_params(**changes), dtype=torch.float32, device="cpu")      # noqa: E731
    for changes, text in (({"window": 5}, "window"), ({"value_dim": 8}, "keys' size"), ({"rotation": "sideways"}, "rotation"),
                          ({"qk_norm_over": "head", "position": PartSpec("none", {"max_positions": 64})}, "whole projection"),
                          ({"gate": "tanh"}, "gate")):
        with pytest.raises(ValueError, match=text):
            build(**changes)


# ---------------------------------------------------------------------- chunks on the host side -- #
def test_the_pages_of_a_chunk_go_back_once_it_is_passed():
    """Chunks of 10 positions on pages of 4: a page is given back when no later query can see any of it; a page that a
    chunk's border cuts stays until the chunk it ends in is passed too."""
    groups, _ = plan_groups([CacheNeed("chunk", 2, 16, chunk=10), CacheNeed("full", 2, 16), CacheNeed("chunk", 2, 16, chunk=10),
                             CacheNeed("chunk", 2, 16, chunk=6)])
    assert [group.entries for group in groups] == [(0, 2), (1,), (3,)]
    assert [group.window for group in groups] == [10, 0, 6]
    manager = CacheManager(groups, page_size=4, num_pages=[8, 16, 8], max_num_seqs=2, max_seq_len=64)
    manager.admit("a")
    kept = {}
    for count in range(1, 33):
        assert manager.reserve("a", count)
        manager.release_passed("a")
        manager.check()
        for group, chunk in ((0, 10), (2, 6)):
            pages = manager.pages_of("a")[group]
            first = count // chunk * chunk             # the next query, at position `count`, sees from here on
            assert [page != 0 for page in pages] == [index * 4 + 3 >= first for index in range(len(pages))], (count, group)
        kept[count] = sum(page != 0 for page in manager.pages_of("a")[0])
    assert kept[9] == 3 and kept[10] == 1 and kept[19] == 3 and kept[20] == 0      # 20 is a border of pages and chunks
    assert all(page != 0 for page in manager.pages_of("a")[1])
    manager.release("a")
    assert [pool.num_held for pool in manager.pools] == [0, 0, 0]
    with pytest.raises(ValueError, match="chunk >= 1"):
        plan_groups([CacheNeed("chunk", 1, 16)])


def test_a_chunk_bounds_the_key_ranges_and_orders_the_tiles():
    """Decode key ranges are laid out for the keys a token sees, not for its whole context; a long prompt's tiles are
    listed by the keys they walk; every row is still covered once per range."""
    far = StepShape(np.ones(2, np.int32), np.array([40_000, 39_999 + 128], np.int32), decode_only=True, page_size=16)
    whole, chunked = AttentionItems(4, 2, 128).plan(far), AttentionItems(4, 2, 128, chunk=256).plan(far)
    assert whole["splits"] > chunked["splits"] == 2             # 65 and 192 keys: two blocks of 128 hold them
    assert AttentionItems(4, 2, 64, chunk=100).plan(far)["splits"] <= 2
    prompt = StepShape(np.array([600], np.int32), np.array([50], np.int32), decode_only=False, page_size=16)
    planner = AttentionItems(4, 2, 128, chunk=200)
    plan = planner.plan(prompt)
    rows = plan["chunk_rows"]
    first = 50 + plan["chunk_items"][:, 1] // 4
    walked = 50 + (plan["chunk_items"][:, 1] + rows) // 4 - first // 200 * 200
    assert sorted(plan["chunk_items"][:, 1].tolist()) == list(range(0, 2400, rows))
    assert (np.diff(walked) <= 0).all()
    assert AttentionItems(4, 2, 128).key != planner.key


def test_the_banded_frequencies_part_follows_the_plain_rule():
    for dims, base, scaling in ((16, 100.0, BANDS), (128, 5.0e5, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}),
                                (32, 1.0e4, {"factor": 2.0, "low": 0.5, "high": 8.0, "original": 20}),
                                (8, 50.0, {"factor": 4.0, "low": 2.0, "high": 2.0, "original": 100})):
        part = POSITION_ENCODINGS.build(BidetarConfig.from_dict(make_config([layer(rot_dims=dims, dim=max(dims, 16), base=base, scaling=scaling)])
                                                                ).to_spec().layers[0].mixer.params["position"], dtype=torch.float32, device="cpu")
        want = torch.tensor(frequencies(dims, base, scaling), dtype=torch.float64)
        torch.testing.assert_close(part.inv_freq.double(), want, rtol=1e-6, atol=0.0)
        plain = torch.tensor(frequencies(dims, base, None), dtype=torch.float64)
        assert (want <= plain * (1 + 1e-12)).all() and (want >= plain / scaling["factor"] * (1 - 1e-12)).all()
    # the three bands of one set: kept, in between, divided
    ratio = torch.tensor(frequencies(16, 100.0, BANDS)) / torch.tensor(frequencies(16, 100.0, None))
    assert float(ratio[0]) == 1.0 and abs(float(ratio[-1]) - 1 / BANDS["factor"]) < 1e-6
    assert any(1 / BANDS["factor"] + 1e-3 < float(value) < 1 - 1e-3 for value in ratio)


# ----------------------------------------------------------- second forms of the plain equations -- #
def test_the_mixer_key_by_key():
    """One query at a time with an explicit list of the keys it sees, the sink as one more term, the gate and the output
    projection head by head."""
    config = CONFIGS["mixer"]
    sizes, weights = config["layers"][0]["mixer"], as_double(make_weights(config, seed=4))
    h = torch.randn(30, config["width"], generator=torch.Generator().manual_seed(2), dtype=torch.float64)
    want = attention_mixer(h, weights, "l0.mix.", sizes, 1e-5)
    H, G, dim, chunk = sizes["heads"], sizes["kv_heads"], sizes["dim"], sizes["mask"]["size"]
    keys, values = keys_and_values(h, weights, "l0.mix.", sizes, 1e-5)
    projected = h @ weights["l0.mix.k"].T + weights["l0.mix.k.b"]
    assert torch.equal(values.reshape(30, -1), projected)
    freq = frequencies(sizes["rot"]["dims"], sizes["rot"]["base"], None)
    q = rms_norm(h @ weights["l0.mix.q"].T + weights["l0.mix.q.b"], weights["l0.mix.q.norm"], 1e-5).view(30, H, dim)
    q = rotate_neighbours(q, sizes["rot"]["dims"], freq)
    out = weights["l0.mix.o"].view(-1, H, dim)
    for i in range(30):
        row = weights["l0.mix.o.b"].clone()
        for head in range(H):
            seen = [j for j in range(30) if j <= i and j // chunk == i // chunk]
            scores = [float(q[i, head] @ keys[j, head // (H // G)]) * sizes["scale"] for j in seen]
            total = math.exp(float(weights["l0.mix.sink"][head])) + sum(math.exp(s) for s in scores)
            mixed = sum(math.exp(s) / total * values[j, head // (H // G)] for s, j in zip(scores, seen))
            gate = 1.0 / (1.0 + math.exp(-float(h[i] @ weights["l0.mix.g"][head])))
            row += out[:, head] @ (gate * mixed)
        assert torch.allclose(row, want[i], atol=1e-9)


def test_the_rotation_by_complex_numbers():
    rows = torch.randn(9, 2, 12, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    freq = frequencies(8, 50.0, BANDS)
    pairs = torch.view_as_complex(rows[..., :8].reshape(9, 2, 4, 2).contiguous())
    turned = pairs * torch.exp(1j * torch.arange(9)[:, None, None] * torch.tensor(freq)[None, None, :])
    want = torch.cat([torch.view_as_real(turned).reshape(9, 2, 8), rows[..., 8:]], dim=-1)
    assert torch.allclose(rotate_neighbours(rows, 8, freq), want)


MECHANISMS = {
    "sink": lambda config, weights: weights.update({n: torch.full_like(w, -1e30) for n, w in weights.items() if n.endswith("sink")}),
    "q bias": lambda config, weights: weights.update({n: 0 * w for n, w in weights.items() if n.endswith("mix.q.b")}),
    "k bias": lambda config, weights: weights.update({n: 0 * w for n, w in weights.items() if n.endswith("mix.k.b")}),
    "o bias": lambda config, weights: weights.update({n: 0 * w for n, w in weights.items() if n.endswith("mix.o.b")}),
    "gate": lambda config, weights: weights.update({n: 0 * w for n, w in weights.items() if n.endswith("mix.g")}),
    "norm weights": lambda config, weights: weights.update({n: torch.ones_like(w) for n, w in weights.items() if n.endswith(".norm")}),
    "residual_mult": lambda config, weights: config.update(residual_mult=1.0),
    "embedding scale": lambda config, weights: config.update(embedding={"scale": 1.0}),
    "one pass": lambda config, weights: config["loop"].update(times=1),
    "feed-forward": lambda config, weights: weights.update({n: 0 * w for n, w in weights.items() if n.endswith("mlp.up")}),
    "no chunks": lambda config, weights: [each["mixer"].pop("mask", None) for each in config["layers"]],
    "chunks one longer": lambda config, weights: [each["mixer"]["mask"].update(size=each["mixer"]["mask"]["size"] + 1)
                                                  for each in config["layers"] if "mask" in each["mixer"]],
    "no bands": lambda config, weights: [each["mixer"].get("rot", {}).pop("scaling", None) for each in config["layers"]],
    "no rotation": lambda config, weights: [each["mixer"].pop("rot", None) for each in config["layers"]],
    "scale": lambda config, weights: [each["mixer"].update(scale=1.1 * each["mixer"]["scale"]) for each in config["layers"]],
}


@pytest.mark.parametrize("what", list(MECHANISMS))
def test_every_mechanism_moves_the_logits(what):
    config = copy.deepcopy(CONFIGS["stack"])
    weights = as_double(make_weights(config, seed=6))
    tokens = torch.randint(0, config["vocab"], (60,), generator=torch.Generator().manual_seed(3)).tolist()
    before = forward(config, weights, tokens)
    MECHANISMS[what](config, weights)
    moved = (forward(config, weights, tokens) - before).pow(2).mean(-1).sqrt()
    assert float(moved[-20:].max()) > 2e-2 * float(before.std()), f"{what} hardly matters to the test model"


def test_mistakes_that_a_plain_comparison_must_show(monkeypatch):
    """Values taken after the norm, halves rotated instead of neighbours, the norm per head, a window in place of chunks:
    each planted in the plain implementation, each moves the logits."""
    config = CONFIGS["stack"]
    weights = as_double(make_weights(config, seed=6))
    tokens = torch.randint(0, config["vocab"], (60,), generator=torch.Generator().manual_seed(3)).tolist()
    before = forward(config, weights, tokens)

    def moved():
        return float((forward(config, weights, tokens) - before).pow(2).mean(-1).sqrt().max() / before.std())

    exact = plain_bidetar.keys_and_values
    monkeypatch.setattr(plain_bidetar, "keys_and_values", lambda *a: (lambda kv: (kv[0], kv[0]))(exact(*a)))
    assert moved() > 0.05
    monkeypatch.setattr(plain_bidetar, "keys_and_values", exact)

    def halves(rows, dims, freq):
        order = list(range(0, dims, 2)) + list(range(1, dims, 2)) + list(range(dims, rows.shape[-1]))
        back = torch.argsort(torch.tensor(order))
        spread = rows.clone()
        spread[..., :dims] = rows[..., back[:dims]] if dims else rows[..., :0]
        return exact_rotation(spread, dims, freq)[..., torch.tensor(order)]

    exact_rotation = plain_bidetar.rotate_neighbours
    monkeypatch.setattr(plain_bidetar, "rotate_neighbours", halves)
    assert moved() > 0.05
    monkeypatch.setattr(plain_bidetar, "rotate_neighbours", exact_rotation)

    def window(T, chunk):
        i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
        return (j <= i) & ((i - j < chunk) if chunk else True)

    exact_mask = plain_bidetar.visible_keys
    monkeypatch.setattr(plain_bidetar, "visible_keys", window)
    assert moved() > 0.05
    monkeypatch.setattr(plain_bidetar, "visible_keys", exact_mask)
    assert moved() == 0.0
