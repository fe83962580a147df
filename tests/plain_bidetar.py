"""A plain, slow restatement of the Bidetar decoder in float64: one function per mechanism, whole sequences only,
no cache, no state, no batch.  It shares no code with the engine; the engine's tests compare against it.

Notation: ``x [T, W]`` rows of one sequence at positions ``0 .. T-1``; weights are ``[out, in]`` and applied as
``x @ W.T``; ``tensors`` maps checkpoint names to float64 tensors.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


# ---------------------------------------------------------------- norms -- #
def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


# ------------------------------------------------------------- rotation -- #
def frequencies(dims: int, base: float, scaling: dict | None) -> list[float]:
    """``f_i = base^(-2i / dims)``, stretched where the wavelength ``2 pi / f`` is long against the original context."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            factor, low, high = (float(scaling[key]) for key in ("factor", "low", "high"))
            original = float(scaling["original"])
            wave = 2.0 * math.pi / f
            if wave < original / high:
                pass
            elif wave > original / low:
                f = f / factor
            else:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate_neighbours(rows: torch.Tensor, dims: int, freq: list[float]) -> torch.Tensor:
    """Rotate the first ``dims`` entries of ``rows [T, heads, n]``: entries ``2i`` and ``2i + 1`` of the row at position
    ``p`` turn by ``p * freq[i]``."""
    if dims == 0:
        return rows
    angle = torch.arange(rows.shape[0], dtype=F64)[:, None] * torch.tensor(freq, dtype=F64)[None, :]
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    u, v = rows[..., 0:dims:2], rows[..., 1:dims:2]
    out = rows.clone()
    out[..., 0:dims:2], out[..., 1:dims:2] = u * cos - v * sin, v * cos + u * sin
    return out


# ------------------------------------------------------------ attention -- #
def visible_keys(T: int, chunk: int) -> torch.Tensor:
    """``[T, T]``: position ``i`` sees ``j <= i`` of its own chunk (``chunk`` 0: of the whole sequence)."""
    seen = torch.zeros(T, T, dtype=torch.bool)
    for i in range(T):
        first = i // chunk * chunk if chunk else 0
        seen[i, first : i + 1] = True
    return seen


def sink_softmax(scores: torch.Tensor, seen: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """``scores [H, T, T]`` to weights ``exp(s) / (exp(sink_h) + sum of exp(s) over the keys seen)``."""
    scores = scores.masked_fill(~seen[None], -math.inf)
    column = sink[:, None, None].expand(-1, scores.shape[1], 1)
    return torch.softmax(torch.cat([scores, column], dim=-1), dim=-1)[..., :-1]


def keys_and_values(h, tensors, prefix: str, sizes: dict, eps: float):
    """``(keys, values)``, both ``[T, G, dim]``: the values are the projected keys, the keys are normed over the whole
    projection and rotated."""
    T, G, dim = h.shape[0], sizes["kv_heads"], sizes["dim"]
    rot = sizes.get("rot") or {}
    dims = int(rot.get("dims", 0))
    projected = h @ tensors[prefix + "k"].T + tensors[prefix + "k.b"]
    normed = rms_norm(projected, tensors[prefix + "k.norm"], eps).view(T, G, dim)
    freq = frequencies(dims, float(rot.get("base", 1.0)), rot.get("scaling"))
    return rotate_neighbours(normed, dims, freq), projected.view(T, G, dim)


def attention_mixer(h, tensors, prefix: str, sizes: dict, eps: float) -> torch.Tensor:
    T, H, G, dim = h.shape[0], sizes["heads"], sizes["kv_heads"], sizes["dim"]
    rot = sizes.get("rot") or {}
    dims = int(rot.get("dims", 0))
    q = rms_norm(h @ tensors[prefix + "q"].T + tensors[prefix + "q.b"], tensors[prefix + "q.norm"], eps).view(T, H, dim)
    q = rotate_neighbours(q, dims, frequencies(dims, float(rot.get("base", 1.0)), rot.get("scaling")))
    k, v = keys_and_values(h, tensors, prefix, sizes, eps)
    k = k.repeat_interleave(H // G, dim=1)       # query head h reads key/value head h // (H / G)
    v = v.repeat_interleave(H // G, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * float(sizes["scale"])
    weights = sink_softmax(scores, visible_keys(T, int((sizes.get("mask") or {}).get("size", 0))), tensors[prefix + "sink"])
    mixed = torch.einsum("hij,jhd->ihd", weights, v)
    mixed = mixed * torch.sigmoid(h @ tensors[prefix + "g"].T)[:, :, None]      # one number a head
    return mixed.reshape(T, H * dim) @ tensors[prefix + "o"].T + tensors[prefix + "o.b"]


# --------------------------------------------------------- feed-forward -- #
def squared_relu_ff(h, tensors, prefix: str) -> torch.Tensor:
    return torch.clamp(h @ tensors[prefix + "up"].T, min=0.0) ** 2 @ tensors[prefix + "down"].T


# ---------------------------------------------------------------- model -- #
def run_order(count: int, loop: dict | None) -> list[int]:
    """Layer indices in the order they run: ``start .. stop - 1`` ``times`` times in a row."""
    if not loop:
        return list(range(count))
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    return list(range(start)) + list(range(start, stop)) * times + list(range(stop, count))


def forward(config: dict, tensors: dict, tokens, collect_layers: bool = False):
    """Logits ``[T, vocab]`` of one sequence (and, with ``collect_layers``, the stream after every layer run)."""
    eps, mult = float(config["norm"]["eps"]), float(config["residual_mult"])
    x = tensors["embed"][torch.as_tensor(tokens)] * float(config["embedding"]["scale"])
    streams = []
    for index in run_order(len(config["layers"]), config.get("loop")):
        layer, p = config["layers"][index], f"l{index}."
        h = rms_norm(x, tensors[p + "norm1"], eps)
        y = attention_mixer(h, tensors, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + squared_relu_ff(h, tensors, p + "mlp.")
        x = x + mult * y
        streams.append(x)
    logits = rms_norm(x, tensors["final.norm"], eps) @ tensors["head"].T
    return (logits, streams) if collect_layers else logits


def greedy(config: dict, tensors: dict, prompt, count: int) -> list[int]:
    tokens = list(prompt)
    for _ in range(count):
        tokens.append(int(forward(config, tensors, tokens)[-1].argmax()))
    return tokens[len(prompt):]
