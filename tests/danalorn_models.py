"""Small Danalorn configurations and seeded weights for the tests.

The weights are drawn so that every mechanism carries weight: token-pair rows of the token rows' size, biases of the
projections' size, sharp scores, sinks of a score's size, gates away from one half, decays from about one half to nearly one.
Every value is rounded to bfloat16 once, so a folder written in either precision and the float64 plain implementation hold
the same numbers.  ``decay_rank`` stands in the configurations here and is left out of the files (a rank is a tensor's shape).
"""

from __future__ import annotations

import copy
import json
import math
from pathlib import Path

import torch


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def latent_layer(*, heads=3, dim=12, rot_dim=8, vdim=10, kv_rank=20, q_rank=18, base=200.0, window=14, scale=0.3,
                 kv_from=None, mlp=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
             "rot": {"base": base, "dims": rot_dim}, "scale": scale}
    if window:
        mixer["mask"] = {"size": window}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def attention_layer(*, heads=6, kv_heads=2, dim=16, vdim=12, scale=0.4, temp=(0.6, 9), mlp=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        mixer["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def gla_layer(*, heads=3, dim=8, vdim=12, tau=6.0, rank=5, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}, "mlp": mlp}


def make_config(layers, *, width=48, vocab=97, eps=1e-5, scale=1.5, buckets=53, mul_prev=11, mul_cur=3) -> dict:
    return {"architecture": "Danalorn", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "layers": copy.deepcopy(list(layers))}


CONFIGS = {
    # one mechanism a model
    "latent": make_config([latent_layer()]),
    "latent, all keys": make_config([latent_layer(window=0, heads=2, mlp=dense())], width=40),
    # readers of a layer's rows: with its window, with a wider one and without one; heads and sizes of their own
    "shared rows": make_config([latent_layer(window=9), latent_layer(kv_from=0, window=21, heads=2, dim=16, vdim=6, q_rank=9, mlp=dense(24)),
                                latent_layer(kv_from=0, window=9, base=200.0, scale=0.2), latent_layer(kv_rank=24, window=5),
                                latent_layer(kv_from=3, kv_rank=24, window=0, heads=4)]),
    "attention": make_config([attention_layer()]),
    "attention, one head a key head": make_config([attention_layer(heads=3, kv_heads=3, dim=8, vdim=24, temp=(0.3, 1), mlp=dense(33))], width=36),
    "attention, no temperature": make_config([attention_layer(heads=4, kv_heads=1, dim=20, vdim=20, temp=None)], width=40),
    "gla": make_config([gla_layer()]),
    "gla, tau one": make_config([gla_layer(heads=2, dim=16, vdim=16, tau=1.0, rank=1, mlp=dense(16))], width=32),
    # everything in one stack, layers with and without a feed-forward
    "stack": make_config([
        gla_layer(mlp=dense(48)), latent_layer(window=12, mlp=dense()), attention_layer(mlp=None), latent_layer(kv_from=1, window=17, heads=2, mlp=dense(30)),
        gla_layer(heads=2, dim=12, vdim=8, tau=16.0, rank=9), attention_layer(heads=4, kv_heads=4, dim=12, vdim=16, temp=(0.5, 16), mlp=dense(64)),
    ], width=64, vocab=120, eps=1e-6, scale=3.0),
    # no size is a multiple of 4
    "narrow": make_config([
        latent_layer(heads=3, dim=7, rot_dim=6, vdim=5, kv_rank=13, q_rank=11, window=3, mlp=dense(27)),
        gla_layer(heads=5, dim=7, vdim=9, tau=2.5, rank=3, mlp=dense(21)),
        latent_layer(heads=1, dim=5, rot_dim=6, vdim=9, kv_rank=13, q_rank=7, window=1, kv_from=0),
        attention_layer(heads=6, kv_heads=3, dim=10, vdim=14, temp=(0.4, 5), mlp=dense(19)),
    ], width=50, vocab=83, buckets=1, mul_prev=1, mul_cur=1),
    # heads of 128 (the tcgen05 tiles), a cached row of 128, recurrent heads of 64
    "wide heads": make_config([
        attention_layer(heads=4, kv_heads=2, dim=128, vdim=128, scale=0.12, temp=(0.5, 32), mlp=dense(160)),
        latent_layer(heads=5, dim=32, rot_dim=32, vdim=24, kv_rank=80, q_rank=64, window=40, scale=0.15),
        gla_layer(heads=2, dim=64, vdim=64, tau=8.0, rank=24),
    ], width=96, vocab=110),
}


def bare(config: dict) -> dict:
    """The configuration as a file holds it."""
    out = copy.deepcopy(config)
    for layer in out["layers"]:
        layer["mixer"].pop("decay_rank", None)
    return out


def tensor_shapes(config: dict) -> dict[str, tuple[int, ...]]:
    width = config["width"]
    shapes = {"embed": (config["vocab"], width), "final.norm": (width,), "head": (config["vocab"], width)}
    if config["embedding"].get("bigram"):
        shapes["bigram"] = (config["embedding"]["bigram"]["buckets"] + 1, width)
    for index, layer in enumerate(config["layers"]):
        p, m = f"l{index}.", layer["mixer"]
        x = p + "mix."
        h = m["heads"]
        shapes.update({p + "norm1": (width,), p + "norm1b": (width,)})
        if layer["type"] == "latent_attention":
            shapes.update({x + "dq": (m["q_rank"], width), x + "dq.norm": (m["q_rank"],), x + "uq": (h * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                           x + "uk": (h * m["dim"], m["kv_rank"]), x + "uv": (h * m["vdim"], m["kv_rank"]), x + "sink": (h,),
                           x + "o": (width, h * m["vdim"])})
            if m.get("kv_from") is None:
                shapes.update({x + "dkv": (m["kv_rank"] + m["rot_dim"], width), x + "dkv.norm": (m["kv_rank"],)})
        elif layer["type"] == "attention":
            q, k, v = h * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            shapes.update({x + "q": (q, width), x + "q.b": (q,), x + "k": (k, width), x + "k.b": (k,), x + "v": (v, width), x + "v.b": (v,),
                           x + "q.norm": (m["dim"],), x + "k.norm": (m["dim"],), x + "g": (h * m["vdim"], width), x + "o": (width, h * m["vdim"])})
        else:
            q, v = h * m["dim"], h * m["vdim"]
            shapes.update({x + "q": (q, width), x + "k": (q, width), x + "v": (v, width), x + "g": (v, width), x + "o": (width, v),
                           x + "norm": (m["vdim"],), x + "a1": (m["decay_rank"], width), x + "a2": (q, m["decay_rank"]), x + "a2.b": (q,)})
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            shapes.update({p + "norm2": (width,), p + "norm2b": (width,), p + "mlp.up": (ff, width), p + "mlp.down": (width, ff)})
    return shapes


def make_weights(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """Float32 tensors whose values are exact in bfloat16."""
    generator = torch.Generator().manual_seed(seed)
    weights = {}
    for name, shape in tensor_shapes(config).items():
        draw = torch.randn(shape, generator=generator)
        last = name.rsplit(".", 1)[-1]
        if name in ("embed", "bigram"):
            value = draw * (1.0 if name == "embed" else 0.9 * config["embedding"]["scale"])
        elif last in ("norm", "norm1", "norm1b", "norm2", "norm2b"):
            value = 1.0 + 0.25 * draw
        elif name.endswith("a2.b"):
            value = 1.5 + 1.5 * draw
        elif last == "b":
            value = 0.4 * draw
        elif last == "sink":
            value = 1.0 + draw
        elif last in ("uq", "g", "a2"):
            value = 2.0 * draw / math.sqrt(shape[-1])
        else:
            value = draw / math.sqrt(shape[-1])
        weights[name] = value.to(torch.bfloat16).to(torch.float32)
    return weights


def write_folder(folder: Path, config: dict, weights: dict[str, torch.Tensor], dtype: torch.dtype) -> Path:
    from rapid_llm_b200.weights.safetensors_io import write_safetensors

    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(bare(config)))
    write_safetensors(folder / "model.safetensors", {name: value.to(dtype) for name, value in weights.items()})
    return folder


def as_double(weights: dict[str, torch.Tensor]) -> dict[str, torch.Tensor]:
    return {name: value.double() for name, value in weights.items()}
