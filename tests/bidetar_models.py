"""Small Bidetar configurations and seeded weights for the tests.

The weights are drawn so that every mechanism carries weight: biases of the projections' size, norm weights spread around
one, sharp attention, sinks of a score's size, gates away from one half.  Every value is rounded to bfloat16 once, so a
folder written in either precision and the float64 plain implementation hold the same numbers.
"""

from __future__ import annotations

import copy
import json
import math
from pathlib import Path

import torch

BANDS = {"factor": 6.0, "low": 1.0, "high": 3.0, "original": 48}


def layer(*, heads=4, kv_heads=2, dim=16, chunk=12, rot_dims=16, base=100.0, scaling=None, scale=0.3, ff=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if chunk:
        mixer["mask"] = {"size": chunk}
    if rot_dims:
        mixer["rot"] = {"base": base, "dims": rot_dims}
        if scaling:
            mixer["rot"]["scaling"] = dict(scaling)
    return {"type": "attention", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def make_config(layers, *, width=64, vocab=97, eps=1e-5, embedding_scale=0.7, residual_mult=0.6, loop=None) -> dict:
    config = {"architecture": "Bidetar", "vocab": vocab, "width": width, "norm": {"eps": eps},
              "embedding": {"scale": embedding_scale}, "residual_mult": residual_mult, "layers": copy.deepcopy(list(layers))}
    if loop is not None:
        config["loop"] = dict(zip(("start", "stop", "times"), loop))
    return config


CONFIGS = {
    # the mixer alone, chunks that neither a page nor a block of keys divides
    "mixer": make_config([layer()]),
    # both sublayers behind one norm, every earlier key visible, banded frequencies on a part of the head
    "parallel": make_config([layer(chunk=0, rot_dims=8, scaling=BANDS, ff=72)], width=48, vocab=61, residual_mult=1.3),
    # a layer before a looped pair and none behind it
    "loop": make_config([layer(ff=40), layer(heads=2, kv_heads=1, dim=32, chunk=7, rot_dims=32, scaling=BANDS), layer(chunk=20, ff=24)],
                        width=40, vocab=70, loop=(1, 3, 3), embedding_scale=1.0),
    # layers that differ in everything: head counts (one kv head, as many as heads), head sizes, chunks, rotated share
    # (none, some, all), bands, feed-forward sizes and none; the loop over the first two
    "stack": make_config([
        layer(heads=6, kv_heads=3, dim=16, chunk=9, rot_dims=4, ff=100),
        layer(heads=4, kv_heads=1, dim=32, chunk=33, rot_dims=32, base=5.0e3, scaling=BANDS, scale=0.2),
        layer(heads=3, kv_heads=3, dim=48, chunk=0, rot_dims=0, scale=0.15, ff=48),
        layer(heads=8, kv_heads=2, dim=16, chunk=16, rot_dims=16, scaling={"factor": 2.0, "low": 0.5, "high": 8.0, "original": 20}, ff=16),
    ], width=72, vocab=130, residual_mult=0.45, loop=(0, 2, 2)),
    # nothing is a multiple of 4 or 8: heads laid out with padding, a width the tensor-core products refuse, chunks of
    # three, of one and of five positions
    "narrow": make_config([
        layer(heads=3, kv_heads=3, dim=10, chunk=3, rot_dims=6, scale=0.7, ff=22),
        layer(heads=5, kv_heads=1, dim=6, chunk=1, rot_dims=2, scale=0.7, ff=13),
        layer(heads=6, kv_heads=2, dim=14, chunk=5, rot_dims=14, scaling=BANDS, scale=0.4),
    ], width=50, vocab=83, eps=1e-6, embedding_scale=1.3, residual_mult=0.9, loop=(2, 3, 2)),
    # heads of 128: the tcgen05 tiles
    "wide heads": make_config([layer(heads=4, kv_heads=2, dim=128, chunk=40, rot_dims=128, base=1.0e4, scaling=BANDS, scale=0.09, ff=160)],
                              width=96, vocab=110, loop=(0, 1, 2)),
}


def tensor_shapes(config: dict) -> dict[str, tuple[int, ...]]:
    width = config["width"]
    shapes = {"embed": (config["vocab"], width), "final.norm": (width,), "head": (config["vocab"], width)}
    for index, each in enumerate(config["layers"]):
        p, m = f"l{index}.", each["mixer"]
        q, k = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
        shapes.update({p + "norm1": (width,), p + "mix.q": (q, width), p + "mix.q.b": (q,), p + "mix.k": (k, width),
                       p + "mix.k.b": (k,), p + "mix.q.norm": (q,), p + "mix.k.norm": (k,), p + "mix.sink": (m["heads"],),
                       p + "mix.g": (m["heads"], width), p + "mix.o": (width, q), p + "mix.o.b": (width,)})
        if each.get("mlp") is not None:
            ff = each["mlp"]["ff"]
            shapes.update({p + "mlp.up": (ff, width), p + "mlp.down": (width, ff)})
    return shapes


def make_weights(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """Float32 tensors whose values are exact in bfloat16."""
    generator = torch.Generator().manual_seed(seed)
    weights = {}
    for name, shape in tensor_shapes(config).items():
        draw = torch.randn(shape, generator=generator)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            value = draw
        elif last == "b":
            value = 0.4 * draw
        elif last in ("norm1", "norm"):
            value = 1.0 + 0.25 * draw
        elif last == "sink":
            value = 1.0 + draw
        elif last == "g":
            value = 2.0 * draw / math.sqrt(shape[-1])
        else:
            value = draw / math.sqrt(shape[-1])
        weights[name] = value.to(torch.bfloat16).to(torch.float32)
    return weights


def write_folder(folder: Path, config: dict, weights: dict[str, torch.Tensor], dtype: torch.dtype) -> Path:
    from rapid_llm_b200.weights.safetensors_io import write_safetensors

    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config))
    write_safetensors(folder / "model.safetensors", {name: value.to(dtype) for name, value in weights.items()})
    return folder


def as_double(weights: dict[str, torch.Tensor]) -> dict[str, torch.Tensor]:
    return {name: value.double() for name, value in weights.items()}
