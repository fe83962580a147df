"""Danalorn's configuration on the CPU: parts and their parameters, expected tensors, the decay's rank from the file, the run
order and the cache groups of layers that read another layer's rows, refusals; the plain implementation against second forms
of the same equations; and that every mechanism of the plain implementation moves the logits of the test models (so a
comparison with it has teeth)."""

from __future__ import annotations

import copy
import json
import math

import numpy as np
import plain_danalorn
import pytest
import torch
from danalorn_models import (
    CONFIGS, as_double, attention_layer, bare, dense, gla_layer, latent_layer, make_config, make_weights, tensor_shapes, write_folder,
)
from plain_danalorn import (
    attention, channel_decays, forward, gated_linear_attention, latent_attention, latent_rows, query_temperature, rms_norm, rotate_neighbours,
)

from rapid_llm_b200.cache import CacheManager, plan_groups
from rapid_llm_b200.config import DanalornConfig, load_config, resolve_architecture
from rapid_llm_b200.config.danalorn import distance_slopes
from rapid_llm_b200.models.causal_lm import CausalLM
from rapid_llm_b200.parts.attention import AttentionItems
from rapid_llm_b200.parts.base import EMBEDDINGS, MIXERS, StepShape
from rapid_llm_b200.weights import load_weights, write_random_model


def _model(config, dtype=torch.float32):
    return CausalLM(DanalornConfig.from_dict(config).to_spec(), dtype, "cpu")


# ------------------------------------------------------------------------------- configuration -- #
def test_the_registry_finds_the_architecture():
    assert resolve_architecture({"architecture": "Danalorn"}) is DanalornConfig


@pytest.mark.parametrize("name", list(CONFIGS))
def test_the_model_expects_the_files_tensors(name):
    assert {n: tuple(s.shape) for n, s in _model(CONFIGS[name]).tensor_specs().items()} == tensor_shapes(CONFIGS[name])


def test_parts_run_order_and_caches():
    config = CONFIGS["stack"]
    spec = DanalornConfig.from_dict(config).to_spec()
    assert {each.arrangement for each in spec.layers} == {"sandwich"}
    assert [each.mixer.kind for each in spec.layers] == ["gated_linear", "latent_attention", "gqa_attention", "latent_attention", "gated_linear",
                                                         "gqa_attention"]
    assert [entry.cache_from for entry in spec.schedule] == [None, None, None, 1, None, None]
    first, reader = spec.layers[1].mixer.params, spec.layers[3].mixer.params
    assert (first["window"], first["cache_window"], first["shares_cache"], first["rotation"], first["sink"]) == (12, 17, False, "neighbours", True)
    assert (reader["window"], reader["shares_cache"], reader["num_heads"]) == (17, True, 2)
    soft = spec.layers[2].mixer.params
    assert (soft["temperature"], soft["sink_score"], soft["gate"], soft["qkv_bias"], soft["qk_norm"], soft["position"].kind) == (
        (0.6, 9.0), 0.0, "sigmoid", True, True, "none")
    assert soft["slopes"] == distance_slopes(6) and soft["slopes"][-1] == 2.0 ** -8 and soft["slopes"][2] == 2.0 ** -4
    assert spec.layers[4].mixer.params["tau"] == 16.0 and spec.layers[4].mixer.params["decay_rank"] == 9
    assert spec.layers[2].feed_forward is None and spec.layers[0].feed_forward.params["activation"] == "relu_squared"
    assert spec.embedding.kind == "summed_embedding" and spec.embedding.params["scale"] == 3.0
    assert spec.final_norm.params["eps"] == 1e-6 and not spec.final_norm.params.get("unit_offset")
    model = CausalLM(spec, torch.float32, "cpu")
    needs = model.cache_needs()
    assert [None if need is None else (need.kind, need.window) for need in needs] == [
        None, ("window", 17), ("full", 0), None, None, ("full", 0)]
    states = [None if need is None else need.shape for need in model.state_needs()]
    assert states == [(3 * 8 * 12,), None, None, None, (2 * 12 * 8,), None, (1,)]
    assert DanalornConfig.from_dict(DanalornConfig.from_dict(config).to_dict()).to_spec() == spec


def test_a_layer_keeps_what_its_widest_reader_needs():
    spec = DanalornConfig.from_dict(CONFIGS["shared rows"]).to_spec()
    needs = CausalLM(spec, torch.float32, "cpu").cache_needs()
    assert [None if need is None else (need.kind, need.window, need.token_shape) for need in needs] == [
        ("window", 21, (32,)), None, None, ("full", 0, (32,)), None]
    assert [each.mixer.params["window"] for each in spec.layers] == [9, 21, 9, 5, 0]
    groups, _ = plan_groups(needs)
    manager = CacheManager(groups, page_size=4, num_pages=[10, 16], max_num_seqs=1, max_seq_len=64)
    manager.admit("a")
    for count in range(1, 41):
        assert manager.reserve("a", count)
        manager.release_passed("a")
        manager.check()
        pages = manager.pages_of("a")[0]
        # the next query, at position `count`, sees back to count - 20 in the widest reader
        assert [page != 0 for page in pages] == [index * 4 + 3 >= count - 20 for index in range(len(pages))]
        assert all(manager.pages_of("a")[1])


def test_without_a_pair_table_or_a_mask_or_a_scale():
    config = make_config([latent_layer(window=0)])
    del config["embedding"]
    spec = DanalornConfig.from_dict(config).to_spec()
    assert spec.embedding.kind == "token_embedding" and spec.embedding.params["scale"] == 1.0 and spec.embedding.params["opens_stream"]
    assert spec.layers[0].mixer.params["window"] == spec.layers[0].mixer.params["cache_window"] == 0
    assert "bigram" not in CausalLM(spec, torch.float32, "cpu").tensor_specs()


def test_the_rank_of_a_decay_comes_from_the_file(tmp_path):
    config = CONFIGS["stack"]
    weights = make_weights(config, seed=1)
    folder = write_folder(tmp_path / "model", config, weights, torch.float32)
    assert "decay_rank" not in json.dumps(json.loads((folder / "config.json").read_text()))
    loaded = load_config(folder)
    assert loaded.to_spec() == DanalornConfig.from_dict(config).to_spec()
    model = CausalLM(loaded.to_spec(), torch.float32, "cpu")
    assert load_weights(model, folder)["tensors"] == len(weights)
    # where the stacked rows of a gated linear mixer lie: each block from a column of eight, nothing between them
    mixer, m = model.layers[4].mixer, config["layers"][4]["mixer"]
    w = mixer.w_in
    cq, cv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
    for at, name in ((0, "q"), (cq, "k"), (2 * cq, "v"), (mixer.g_col0, "g"), (mixer.a_col0, "a1")):
        rows = weights[f"l4.mix.{name}"]
        assert torch.equal(w[at : at + rows.shape[0]], rows)
    assert mixer.g_col0 % 8 == mixer.a_col0 % 8 == w.shape[0] % 8 == 0
    assert not w[2 * cq + cv : mixer.g_col0].any() and not w[mixer.a_col0 + m["decay_rank"] :].any()
    # the gate's rows of an attention layer ride behind q, k and v and have no bias
    soft, m = model.layers[2].mixer, config["layers"][2]["mixer"]
    assert torch.equal(soft.qkv[soft.qkv_rows : soft.qkv_rows + soft.gate_width].view(m["heads"], soft.d, -1)[:, : m["vdim"]].reshape(-1, 64),
                       weights["l2.mix.g"])
    assert not soft.qkv_bias[soft.qkv_rows :].any() and torch.equal(soft.sink, torch.zeros(m["heads"]))
    # a layer that reads another one's rows has none of its own in its first product
    assert model.layers[3].mixer.down.shape[0] == -(-config["layers"][3]["mixer"]["q_rank"] // 8) * 8
    broken = {name: value for name, value in weights.items() if name != "l4.mix.a1"}
    write_folder(tmp_path / "broken", config, broken, torch.float32)
    with pytest.raises(ValueError, match="l4.mix.a1"):
        load_config(tmp_path / "broken")


def test_a_random_model_folder_round_trip(tmp_path):
    config = DanalornConfig.from_dict(CONFIGS["stack"])
    folder = write_random_model(tmp_path / "model", config, seed=3, dtype=torch.bfloat16)
    loaded = load_config(folder)
    assert isinstance(loaded, DanalornConfig) and loaded.to_spec() == config.to_spec()
    model = CausalLM(loaded.to_spec(), torch.bfloat16, "cpu")
    assert load_weights(model, folder)["tensors"] == len(tensor_shapes(CONFIGS["stack"]))
    used = model.parameter_bytes()
    exact = sum((2 if len(shape) == 2 else 4) * math.prod(shape) for shape in tensor_shapes(CONFIGS["stack"]).values())
    assert exact <= used <= 1.15 * exact          # heads of 12 are laid out in 16, blocks of rows start on eight


def test_refusals():
    def refuse(text, change, name="stack"):
        config = copy.deepcopy(CONFIGS[name])
        change(config)
        with pytest.raises(ValueError, match=text):
            DanalornConfig.from_dict(config)

    refuse("unknown mixer type", lambda c: c["layers"][0].update(type="wkv"))
    refuse("unknown feed-forward kind", lambda c: c["layers"][0]["mlp"].update(kind="moe"))
    refuse("lacks 'tau'", lambda c: c["layers"][0]["mixer"].pop("tau"))
    refuse("lacks 'kv_rank'", lambda c: c["layers"][1]["mixer"].pop("kv_rank"))
    refuse("lacks 'kv_heads'", lambda c: c["layers"][2]["mixer"].pop("kv_heads"))
    refuse("rot.dims", lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4))
    refuse("rot.base", lambda c: c["layers"][1]["mixer"].pop("rot"))
    refuse("earlier latent_attention layer", lambda c: c["layers"][3]["mixer"].update(kv_from=2))
    refuse("earlier latent_attention layer", lambda c: c["layers"][3]["mixer"].update(kv_from=3))
    refuse("must equal layer 1's", lambda c: c["layers"][3]["mixer"].update(kv_rank=24))
    refuse("must equal layer 1's", lambda c: c["layers"][3]["mixer"]["rot"].update(base=300.0))
    refuse("no latent of its own", lambda c: c["layers"][2]["mixer"].update(kv_from=1), "shared rows")
    refuse("lacks 'width'", lambda c: c.pop("width"))
    refuse("at least one layer", lambda c: c.update(layers=[]))

    spec = DanalornConfig.from_dict(CONFIGS["stack"]).to_spec()

    def build(index, **changes):
        return MIXERS.build(spec.layers[index].mixer.with_params(**changes), dtype=torch.float32, device="cpu")

    for index, changes, text in ((1, {"cache_window": 5}, "cache_window"), (1, {"kv_rank": 700}, "640"), (2, {"sink": True}, "learned or fixed"),
                                 (2, {"slopes": [1.0]}, "one number per query head"), (2, {"temperature": (1.0, 0.0)}, "positive"),
                                 (4, {"tau": 0.0}, "positive"), (3, {"q_rank": None}, "query latent")):
        with pytest.raises(ValueError, match=text):
            build(index, **changes)
    with pytest.raises(ValueError, match="pair bucket"):
        EMBEDDINGS.build(spec.embedding.with_params(pair_buckets=0), dtype=torch.float32, device="cpu")


def test_a_window_bounds_the_key_ranges_where_a_mixer_asks():
    far = StepShape(np.ones(1, np.int32), np.array([40_000], np.int32), decode_only=True, page_size=16)
    whole, windowed = AttentionItems(8, 1, 128, tensor_core=False).plan(far), AttentionItems(8, 1, 128, tensor_core=False, window=130).plan(far)
    assert whole["splits"] == 16 and windowed["splits"] == 4
    assert AttentionItems(8, 1, 128).key != AttentionItems(8, 1, 128, window=130).key


# ----------------------------------------------------------- second forms of the plain equations -- #
def _rows(config, count, seed):
    return torch.randn(count, config["width"], generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def test_latent_attention_over_the_cached_rows_alone():
    """Nothing expanded per key: W_uk moved to the queries, W_uv behind the weighted sum of the latents; one query at a time
    with an explicit list of the keys it sees and the sink as one more term."""
    config = CONFIGS["latent"]
    sizes, weights = config["layers"][0]["mixer"], as_double(make_weights(config, seed=4))
    h = _rows(config, 40, 2)
    c, k_rot = latent_rows(h, weights, "l0.mix.", sizes, 1e-5)
    want = latent_attention(h, weights, "l0.mix.", sizes, 1e-5, (c, k_rot))
    H, dim, rot, rank, vdim, window = 3, 12, 8, 20, 10, 14
    uk, uv = weights["l0.mix.uk"].view(H, dim, rank), weights["l0.mix.uv"].view(H, vdim, rank)
    q = (rms_norm(h @ weights["l0.mix.dq"].T, weights["l0.mix.dq.norm"], 1e-5) @ weights["l0.mix.uq"].T).view(40, H, dim + rot)
    q_rot = rotate_neighbours(q[..., dim:], 200.0)
    out = weights["l0.mix.o"].view(-1, H, vdim)
    for i in range(40):
        row = torch.zeros(config["width"], dtype=torch.float64)
        for head in range(H):
            seen = list(range(max(0, i - window + 1), i + 1))
            at_latent = uk[head].T @ q[i, head, :dim]
            terms = [math.exp(0.3 * float(at_latent @ c[j] + q_rot[i, head] @ k_rot[j])) for j in seen]
            total = sum(terms) + math.exp(float(weights["l0.mix.sink"][head]))
            row += out[:, head] @ (uv[head] @ sum(term / total * c[j] for term, j in zip(terms, seen)))
        assert torch.allclose(row, want[i], atol=1e-9)


def test_attention_key_by_key():
    config = CONFIGS["attention"]
    sizes, weights = config["layers"][0]["mixer"], as_double(make_weights(config, seed=4))
    h = _rows(config, 30, 3)
    want = attention(h, weights, "l0.mix.", sizes, 1e-5)
    H, G, dim, vdim = 6, 2, 16, 12
    q, k, v = ((h @ weights[f"l0.mix.{n}"].T + weights[f"l0.mix.{n}.b"]).view(30, heads, size)
               for n, heads, size in (("q", H, dim), ("k", G, dim), ("v", G, vdim)))
    out, gates = weights["l0.mix.o"].view(-1, H, vdim), weights["l0.mix.g"].view(H, vdim, -1)
    for i in range(30):
        row = torch.zeros(config["width"], dtype=torch.float64)
        warm = 1.0 + 0.6 * math.log((i + 1) // 9 + 1)
        for head in range(H):
            query = warm * rms_norm(q[i, head], weights["l0.mix.q.norm"], 1e-5)
            terms = []
            for j in range(i + 1):
                key = rms_norm(k[j, head // 3], weights["l0.mix.k.norm"], 1e-5)
                terms.append(math.exp(0.4 * float(query @ key) - 2.0 ** (-8.0 * (head + 1) / H) * (i - j)))
            mixed = sum(term * v[j, head // 3] for j, term in enumerate(terms)) / (1.0 + sum(terms))
            row += out[:, head] @ (mixed / (1.0 + torch.exp(-gates[head] @ h[i])))
        assert torch.allclose(row, want[i], atol=1e-9)


def test_the_temperature_steps_where_a_stretch_is_full():
    values = query_temperature(40, 0.5, 16).tolist()
    assert values[:15] == [1.0] * 15 and values[15] == values[30] == 1.0 + 0.5 * math.log(2.0) and values[31] == 1.0 + 0.5 * math.log(3.0)


def test_gated_linear_attention_as_a_sum_over_earlier_tokens():
    """``o_t = sum_j (prod of the decays behind j up to t) . k_j . q_t / sqrt(dim) v_j``; the decay as the exponential of a
    scaled softplus; the queries' factor moved into the norm's eps."""
    config = CONFIGS["gla"]
    sizes, weights = config["layers"][0]["mixer"], as_double(make_weights(config, seed=4))
    h = _rows(config, 25, 5)
    want = gated_linear_attention(h, weights, "l0.mix.", sizes, 1e-5)
    H, dim, vdim = 3, 8, 12
    z = (h @ weights["l0.mix.a1"].T) @ weights["l0.mix.a2"].T + weights["l0.mix.a2.b"]
    alpha = torch.exp(-torch.nn.functional.softplus(-z) / 6.0)
    assert torch.allclose(alpha, channel_decays(h, weights, "l0.mix.", 6.0), atol=1e-12)
    alpha = alpha.view(25, H, dim)
    q, k, v = ((h @ weights[f"l0.mix.{n}"].T).view(25, H, size) for n, size in (("q", dim), ("k", dim), ("v", vdim)))
    g = h @ weights["l0.mix.g"].T
    for t in range(25):
        read = torch.zeros(H, vdim, dtype=torch.float64)
        for j in range(t + 1):
            behind = alpha[j + 1 : t + 1].prod(dim=0)
            read += (behind * k[j] * q[t]).sum(-1, keepdim=True) * v[j]
        out = (read / torch.sqrt(read.square().mean(-1, keepdim=True) + 1e-5 * dim) * weights["l0.mix.norm"]).reshape(-1)
        assert torch.allclose((out * torch.nn.functional.silu(g[t])) @ weights["l0.mix.o"].T, want[t], atol=1e-9)


def test_the_rotation_by_complex_numbers():
    rows = _rows({"width": 2 * 12}, 9, 0).view(9, 2, 12)
    pairs = torch.view_as_complex(rows.reshape(9, 2, 6, 2).contiguous())
    freq = torch.tensor([50.0 ** (-2.0 * i / 12) for i in range(6)], dtype=torch.float64)
    turned = pairs * torch.exp(1j * torch.arange(9)[:, None, None] * freq[None, None, :])
    assert torch.allclose(rotate_neighbours(rows, 50.0), torch.view_as_real(turned).reshape(9, 2, 12))


def test_the_pair_rows_by_hand():
    assert plain_danalorn.pair_rows([4, 9, 4], 10, 3, 2) == [10, (4 * 3 + 9 * 2) % 10, (9 * 3 + 4 * 2) % 10]
    assert plain_danalorn.pair_rows([7], 5, 1, 1) == [5]


def _each(kind, change):
    def apply(config, weights):
        for layer in config["layers"]:
            if layer["type"] == kind:
                change(layer["mixer"])
    return apply


def _set(suffix, value):
    return lambda config, weights: weights.update({n: value(w) for n, w in weights.items() if n.endswith(suffix)})


MECHANISMS = {
    "token pairs": _set("bigram", lambda w: 0 * w),
    "the first token's row": lambda config, weights: weights["bigram"].__setitem__(-1, 0.0),
    "embedding scale": lambda config, weights: config["embedding"].update(scale=1.0),
    "closing norms": lambda config, weights: weights.update({n: torch.ones_like(w) for n, w in weights.items() if n.endswith(("norm1b", "norm2b"))}),
    "latent sink": _set("sink", lambda w: w - 1e30),
    "latent query norm": _set("dq.norm", torch.ones_like),
    "latent norm": _set("dkv.norm", torch.ones_like),
    "window": _each("latent_attention", lambda m: m.pop("mask", None)),
    "window one longer": _each("latent_attention", lambda m: m["mask"].update(size=m["mask"]["size"] + 1)),
    "window one shorter": _each("latent_attention", lambda m: m["mask"].update(size=m["mask"]["size"] - 1)),
    "rotation": _each("latent_attention", lambda m: m["rot"].update(base=1e30)),
    "latent scale": _each("latent_attention", lambda m: m.update(scale=1.1 * m["scale"])),
    "temperature": _each("attention", lambda m: m.pop("q_temp", None)),
    "temperature a stretch longer": _each("attention", lambda m: m["q_temp"].update(every=m["q_temp"]["every"] + 1)),
    "q bias": _set("q.b", lambda w: 0 * w),
    "k bias": _set("k.b", lambda w: 0 * w),
    "v bias": _set("v.b", lambda w: 0 * w),
    "head norms": lambda config, weights: weights.update({n: torch.ones_like(w) for n, w in weights.items() if n.endswith(("q.norm", "k.norm"))}),
    "attention scale": _each("attention", lambda m: m.update(scale=1.1 * m["scale"])),
    "gates": _set("mix.g", lambda w: 0.5 * w),
    "tau": _each("gla", lambda m: m.update(tau=1.3 * m["tau"])),
    "decay bias": _set("a2.b", lambda w: w + 0.5),
    "decay from the input": _set("a2", lambda w: 0 * w),
    "recurrent norm": _set("mix.norm", torch.ones_like),
    "feed-forward": _set("mlp.up", lambda w: 0 * w),
}


def _tokens(config, count=60):
    return torch.randint(0, config["vocab"], (count,), generator=torch.Generator().manual_seed(3)).tolist()


@pytest.mark.parametrize("what", list(MECHANISMS))
def test_every_mechanism_moves_the_logits(what):
    config = copy.deepcopy(CONFIGS["stack"])
    weights = as_double(make_weights(config, seed=6))
    tokens = _tokens(config)
    before = forward(tokens, weights, config)
    MECHANISMS[what](config, weights)
    moved = (forward(tokens, weights, config) - before).pow(2).mean(-1).sqrt()
    assert float(moved.max()) > 2e-2 * float(before.std()), f"{what} hardly matters to the test model"


def test_mistakes_that_a_plain_comparison_must_show(monkeypatch):
    """Halves rotated instead of neighbours, a distance taken from the key's position, no fixed sink, a reader that uses its
    own projection, a first token that takes row 0: each planted in the plain implementation, each moves the logits."""
    config = CONFIGS["stack"]
    weights = as_double(make_weights(config, seed=6))
    tokens = _tokens(config)
    before = forward(tokens, weights, config)

    def moved():
        return float((forward(tokens, weights, config) - before).pow(2).mean(-1).sqrt().max() / before.std())

    exact = {name: getattr(plain_danalorn, name) for name in ("rotate_neighbours", "distance_slopes", "weights_with_sink", "latent_rows", "pair_rows")}

    def halves(rows, base):
        R = rows.shape[-1]
        order = torch.tensor(list(range(0, R, 2)) + list(range(1, R, 2)))
        back = torch.argsort(order)
        return exact["rotate_neighbours"](rows[..., back], base)[..., order]

    plants = {
        "rotate_neighbours": halves,
        "distance_slopes": lambda heads: [2.0 ** (-8.0 * head / heads) for head in range(heads)],
        "weights_with_sink": lambda scores, seen, sink: exact["weights_with_sink"](scores, seen, sink - (1e30 if not sink.any() else 0.0)),
        "latent_rows": lambda *a: (lambda c, k: (c, 0 * k))(*exact["latent_rows"](*a)),
        "pair_rows": lambda tokens, buckets, *m: [0] + exact["pair_rows"](tokens, buckets, *m)[1:],
    }
    for name, plant in plants.items():
        monkeypatch.setattr(plain_danalorn, name, plant)
        assert moved() > 0.03, name
        monkeypatch.setattr(plain_danalorn, name, exact[name])
    assert moved() == 0.0


def test_the_configuration_of_a_file_holds_no_rank():
    assert "decay_rank" not in json.dumps(bare(make_config([gla_layer(), attention_layer(mlp=dense())])))
