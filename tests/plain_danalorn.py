"""A plain, slow restatement of the Danalorn decoder in float64: one function per mechanism, whole sequences only, no
cache, no state, no batch.  It shares no code with the engine; the engine's tests compare against it.

Notation: ``x [T, W]`` rows of one sequence at positions ``0 .. T-1``; weights are ``[out, in]`` and applied as
``x @ W.T``; ``tensors`` maps checkpoint names to tensors of any dtype; ``config`` is the parsed ``config.json``.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


_STORE = None      # what rounding() does to a number where an engine stores it; None: nothing


def _t(tensors, name):
    return tensors[name].to(F64)


def _stored(x: torch.Tensor) -> torch.Tensor:
    return x if _STORE is None else _STORE(x)


def _linear(x: torch.Tensor, tensors, name: str) -> torch.Tensor:
    return _stored(x @ _t(tensors, name).T)


def over_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.square().mean(-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return over_rms(x, eps) * weight


# ------------------------------------------------------------- embedding -- #
def pair_rows(tokens, buckets: int, mul_prev: int, mul_cur: int) -> list[int]:
    """The row of the pair table every token adds: hashed from the token before it and itself; the extra last row for a
    sequence's first token."""
    rows = [buckets]
    for before, token in zip(tokens, tokens[1:]):
        rows.append((before * mul_prev + token * mul_cur) % buckets)
    return rows[: len(tokens)]


def embed(tokens, tensors, config) -> torch.Tensor:
    tokens = [int(token) for token in tokens]
    section = config["embedding"]
    x = _t(tensors, "embed")[tokens] * float(section.get("scale", 1.0))
    pair = section.get("bigram")
    if pair:
        x = x + _t(tensors, "bigram")[pair_rows(tokens, pair["buckets"], pair["mul_prev"], pair["mul_cur"])]
    return x


# ------------------------------------------------------------- rotation -- #
def rotate_neighbours(x: torch.Tensor, base: float) -> torch.Tensor:
    """``x [T, ..., R]``: entries ``2i`` and ``2i + 1`` of the row at position ``p`` turn by ``p base^(-2i / R)``."""
    T, R = x.shape[0], x.shape[-1]
    out = torch.empty_like(x)
    for i in range(R // 2):
        angle = torch.arange(T, dtype=F64) * float(base) ** (-2.0 * i / R)
        shape = [T] + [1] * (x.dim() - 2)
        cos, sin = torch.cos(angle).view(shape), torch.sin(angle).view(shape)
        a, b = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = a * cos - b * sin
        out[..., 2 * i + 1] = b * cos + a * sin
    return out


# ------------------------------------------------------------ visibility -- #
def visible(T: int, window: int) -> torch.Tensor:
    """``[T, T]``: which keys (columns) a query (row) sees; ``window`` 0 = every earlier one and its own."""
    behind = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (behind >= 0) if window <= 0 else (behind >= 0) & (behind < window)


def weights_with_sink(scores: torch.Tensor, seen: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """``scores [H, T, T]``; ``exp(sink[h])`` joins each row's denominator and nothing else."""
    scores = scores.masked_fill(~seen[None], -math.inf)
    extra = sink.to(F64)[:, None, None].expand(-1, scores.shape[1], 1)
    return torch.softmax(torch.cat([scores, extra], dim=-1), dim=-1)[..., :-1]


# ------------------------------------------------------ latent attention -- #
def latent_rows(h, tensors, prefix, sizes, eps):
    """What a layer with a latent of its own caches: ``(c [T, rank], rotated key part [T, rot])``."""
    rank = int(sizes["kv_rank"])
    down = _linear(h, tensors, prefix + "dkv")
    c = _stored(rms_norm(down[:, :rank], _t(tensors, prefix + "dkv.norm"), eps))
    return c, _stored(rotate_neighbours(down[:, rank:], float((sizes.get("rot") or {}).get("base", 1.0))))


def latent_attention(h, tensors, prefix, sizes, eps, source):
    """``source``: the rows of :func:`latent_rows`, this layer's or those of the layer it reads."""
    T = h.shape[0]
    H, dim, rot, vdim = (int(sizes[key]) for key in ("heads", "dim", "rot_dim", "vdim"))
    c, k_rot = source
    c_q = _stored(rms_norm(_linear(h, tensors, prefix + "dq"), _t(tensors, prefix + "dq.norm"), eps))
    q = _linear(c_q, tensors, prefix + "uq").view(T, H, dim + rot)
    q_rot = rotate_neighbours(q[..., dim:], float((sizes.get("rot") or {}).get("base", 1.0)))
    k = _linear(c, tensors, prefix + "uk").view(T, H, dim)
    v = _linear(c, tensors, prefix + "uv").view(T, H, vdim)
    scores = torch.einsum("ihd,jhd->hij", q[..., :dim], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)
    seen = visible(T, int((sizes.get("mask") or {}).get("size", 0)))
    shares = weights_with_sink(scores * float(sizes["scale"]), seen, _t(tensors, prefix + "sink"))
    return _linear(_stored(torch.einsum("hij,jhd->ihd", shares, v).reshape(T, H * vdim)), tensors, prefix + "o")


# ------------------------------------------------------------- attention -- #
def query_temperature(T: int, coef: float, every: float) -> torch.Tensor:
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0) for p in range(T)], dtype=F64)


def distance_slopes(heads: int) -> list[float]:
    return [2.0 ** (-8.0 * (head + 1) / heads) for head in range(heads)]


def attention(h, tensors, prefix, sizes, eps):
    T = h.shape[0]
    H, G, dim, vdim = (int(sizes[key]) for key in ("heads", "kv_heads", "dim", "vdim"))

    def projected(name, heads, size):
        return _stored(h @ _t(tensors, prefix + name).T + _t(tensors, prefix + name + ".b")).view(T, heads, size)

    q = rms_norm(projected("q", H, dim), _t(tensors, prefix + "q.norm"), eps)
    k = rms_norm(projected("k", G, dim), _t(tensors, prefix + "k.norm"), eps)
    v = projected("v", G, vdim)
    warm = sizes.get("q_temp")
    if warm:
        q = q * query_temperature(T, float(warm["coef"]), float(warm["every"]))[:, None, None]
    q, k = _stored(q), _stored(k)
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * float(sizes["scale"])
    behind = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(F64)
    scores = scores - torch.tensor(distance_slopes(H), dtype=F64)[:, None, None] * behind
    shares = weights_with_sink(scores, visible(T, 0), torch.zeros(H, dtype=F64))
    out = torch.einsum("hij,jhd->ihd", shares, v).reshape(T, H * vdim)
    return _linear(_stored(_stored(out) * torch.sigmoid(_linear(h, tensors, prefix + "g"))), tensors, prefix + "o")


# ------------------------------------------------- gated linear attention -- #
def channel_decays(h, tensors, prefix, tau: float) -> torch.Tensor:
    z = _linear(h, tensors, prefix + "a1") @ _t(tensors, prefix + "a2").T + _t(tensors, prefix + "a2.b")
    return torch.sigmoid(z) ** (1.0 / tau)


def gated_linear_attention(h, tensors, prefix, sizes, eps):
    T = h.shape[0]
    H, dim, vdim = (int(sizes[key]) for key in ("heads", "dim", "vdim"))
    q = _linear(h, tensors, prefix + "q").view(T, H, dim) / math.sqrt(dim)
    k = _linear(h, tensors, prefix + "k").view(T, H, dim)
    v = _linear(h, tensors, prefix + "v").view(T, H, vdim)
    alpha = channel_decays(h, tensors, prefix, float(sizes["tau"])).view(T, H, dim)
    S = torch.zeros(H, dim, vdim, dtype=F64)
    read = []
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        read.append(torch.einsum("hkv,hk->hv", S, q[t]))
    out = rms_norm(torch.stack(read), _t(tensors, prefix + "norm"), eps).reshape(T, H * vdim)
    g = _linear(h, tensors, prefix + "g")
    return _linear(_stored(out * g * torch.sigmoid(g)), tensors, prefix + "o")


# ---------------------------------------------------------- feed-forward -- #
def squared_relu_feed_forward(h, tensors, prefix):
    return _linear(_stored(_linear(h, tensors, prefix + "up").clamp(min=0).square()), tensors, prefix + "down")


# -------------------------------------------------------------- the model -- #
def forward(tokens, tensors, config, return_layers: bool = False):
    """Logits ``[T, vocab]`` (float64) of a whole sequence; with ``return_layers`` also the stream after every layer."""
    eps = float(config["norm"]["eps"])
    x = embed(tokens, tensors, config)
    streams, cached = [], {}
    for index, layer in enumerate(config["layers"]):
        p, sizes = f"l{index}.", layer["mixer"]
        h = _stored(rms_norm(x, _t(tensors, p + "norm1"), eps))
        if layer["type"] == "latent_attention":
            source = sizes.get("kv_from")
            if source is None:
                cached[index] = latent_rows(h, tensors, p + "mix.", sizes, eps)
            mixed = latent_attention(h, tensors, p + "mix.", sizes, eps, cached[index if source is None else source])
        elif layer["type"] == "attention":
            mixed = attention(h, tensors, p + "mix.", sizes, eps)
        elif layer["type"] == "gla":
            mixed = gated_linear_attention(h, tensors, p + "mix.", sizes, eps)
        else:
            raise ValueError(layer["type"])
        x = x + rms_norm(mixed, _t(tensors, p + "norm1b"), eps)
        if layer.get("mlp") is not None:
            h = _stored(rms_norm(x, _t(tensors, p + "norm2"), eps))
            x = x + rms_norm(squared_relu_feed_forward(h, tensors, p + "mlp."), _t(tensors, p + "norm2b"), eps)
        streams.append(x)
    logits = _stored(rms_norm(x, _t(tensors, "final.norm"), eps)) @ _t(tensors, "head").T
    return (logits, torch.stack(streams)) if return_layers else logits


def rounding(tokens, tensors, config, dtype: torch.dtype, exact: torch.Tensor, draws: int = 8) -> torch.Tensor:
    """Per row, how far the logits move when every projection, norm and head output passes ``dtype`` where an engine of that
    precision stores it: the root mean square of the difference as a share of the row's own (means removed), the most of one
    rounding and ``draws - 1`` random errors of its size.

    A sublayer's result is normed on its way to the stream, so a result near zero (a read-out whose query hardly meets the
    state, a squared relu with nothing left of its few entries) comes out as large as any other, with a direction that
    rounding decides; a row of that kind says little about an engine in 16 bits."""
    global _STORE
    size = (exact - exact.mean(-1, keepdim=True)).square().mean(-1).sqrt()
    generator = torch.Generator().manual_seed(len(tokens))
    most = torch.zeros_like(size)
    for draw in range(draws):
        if draw == 0:
            _STORE = lambda x: x.to(dtype).to(F64)      # noqa: E731
        else:
            _STORE = lambda x: x * (1.0 + (torch.rand(x.shape, generator=generator, dtype=F64) - 0.5) * torch.finfo(dtype).eps)      # noqa: E731
        try:
            moved = forward(tokens, tensors, config) - exact
        finally:
            _STORE = None
        most = torch.maximum(most, (moved - moved.mean(-1, keepdim=True)).square().mean(-1).sqrt() / size)
    return most


def greedy(tokens, tensors, config, steps: int) -> list[int]:
    """The ``steps`` tokens that always taking the largest logit produces after ``tokens``."""
    tokens = list(tokens)
    start = len(tokens)
    for _ in range(steps):
        tokens.append(int(forward(tokens, tensors, config)[-1].argmax()))
    return tokens[start:]
