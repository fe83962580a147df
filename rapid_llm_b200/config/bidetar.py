"""Configuration of the Bidetar decoder: a list of attention layers with a dense feed-forward (or none) beside the
mixer, part of them run in a loop.

``config.json`` gives ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``residual_mult``, ``loop`` (layers
``start .. stop - 1`` run ``times`` times in a row with the same weights; every pass has a cache of its own; nothing
joins the stream between passes) and ``layers``: one entry a layer, ``type`` names the mixer (``attention``), ``mixer``
its sizes and constants, ``mlp`` the feed-forward (``kind`` ``dense``) or ``null``.  Layer ``i``'s tensors start with
``l<i>.``.

What the parts are built from:

* every layer is the arrangement ``shared_norm``: ``x <- x + m (mixer(n) + ff(n))`` with ``n = norm1(x)``, an RMS norm,
  and ``m = residual_mult``, the norms' ``add_scale``; the scaled embedding opens the float32 stream;
* ``attention`` -> ``gqa_attention``: biases on q, k and the output projection; the projected keys are the values
  (``values_from_keys``); q and k RMS-normed over their whole projection (weights ``q.norm``, ``k.norm``); the first
  ``rot.dims`` entries of a head rotated in neighbouring pairs, with frequencies ``rot.base^(-2i / dims)`` stretched in
  bands where ``rot.scaling`` is given; ``scale`` on the scores; chunks of ``mask.size`` positions (none: every earlier
  position); a sink per head; a gate of one number per head;
* ``dense`` -> ``dense`` with the square of relu;
* the model ends in an RMS norm (``final.norm``) and an untied head.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Mapping

from .model_spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MAX_POSITIONS = 1 << 20     # nothing tabulated bounds a sequence; the engine's max_seq_len does


@dataclass
class BidetarConfig:
    architecture = "Bidetar"
    model_type = "bidetar"

    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    residual_mult: float
    layers: list[dict[str, Any]]
    loop: dict[str, int] | None = None
    raw: dict[str, Any] = field(default_factory=dict)

    # -------------------------------------------------------------- reading #
    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], overrides: Mapping[str, Any] | None = None) -> "BidetarConfig":
        raw = copy.deepcopy(dict(raw))
        raw.update(copy.deepcopy(dict(overrides or {})))
        for key in ("vocab", "width", "layers", "norm"):
            if key not in raw:
                raise ValueError(f"config.json of a Bidetar model lacks {key!r}")
        config = cls(vocab=int(raw["vocab"]), width=int(raw["width"]), norm_eps=float(raw["norm"]["eps"]),
                     embedding_scale=float((raw.get("embedding") or {}).get("scale", 1.0)),
                     residual_mult=float(raw.get("residual_mult", 1.0)), layers=list(raw["layers"]),
                     loop=raw.get("loop") or None, raw=raw)
        config.validate()
        return config

    def validate(self) -> None:
        if not self.layers:
            raise ValueError("a Bidetar model needs at least one layer")
        for index, layer in enumerate(self.layers):
            if layer.get("type") != "attention":
                raise ValueError(f"layer {index}: unknown mixer type {layer.get('type')!r}")
            mixer = layer.get("mixer") or {}
            for key in ("heads", "kv_heads", "dim", "scale"):
                if key not in mixer:
                    raise ValueError(f"layer {index}: the attention mixer lacks {key!r}")
            if int(mixer.get("vdim", mixer["dim"])) != int(mixer["dim"]):
                raise ValueError(f"layer {index}: the values are the projected keys, so vdim ({mixer['vdim']}) must equal dim ({mixer['dim']})")
            if int((mixer.get("mask") or {}).get("size", 0) or 0) < 0:
                raise ValueError(f"layer {index}: mask.size must not be negative")
            scaling = (mixer.get("rot") or {}).get("scaling")
            for key in ("factor", "low", "high", "original") if scaling else ():
                if key not in scaling:
                    raise ValueError(f"layer {index}: rot.scaling lacks {key!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {index}: unknown feed-forward kind {mlp.get('kind')!r}")
        if self.loop:
            start, stop, times = (int(self.loop[key]) for key in ("start", "stop", "times"))
            if not 0 <= start < stop <= len(self.layers) or times < 1:
                raise ValueError(f"loop {self.loop} does not fit {len(self.layers)} layers")

    def to_dict(self) -> dict[str, Any]:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
               "residual_mult": self.residual_mult, "layers": copy.deepcopy(self.layers)}
        if self.loop:
            out["loop"] = dict(self.loop)
        return out

    # ----------------------------------------------------------------- spec #
    def _mixer(self, layer: Mapping[str, Any]) -> PartSpec:
        sizes = layer["mixer"]
        rot = sizes.get("rot") or {}
        frequencies = {"rotary_dim": int(rot.get("dims", 0)), "theta": float(rot.get("base", 10000.0)),
                       "max_positions": MAX_POSITIONS}
        position = PartSpec("rotary_frequencies", frequencies)
        if rot.get("scaling"):
            bands = {key: float(rot["scaling"][key]) for key in ("factor", "low", "high", "original")}
            position = PartSpec("banded_frequencies", {**frequencies, **bands})
        return PartSpec("gqa_attention", {
            "hidden_size": self.width, "num_heads": int(sizes["heads"]), "num_kv_heads": int(sizes["kv_heads"]),
            "head_dim": int(sizes["dim"]), "scale": float(sizes["scale"]), "qkv_bias": True, "o_bias": True,
            "values_from_keys": True, "qk_norm": True, "qk_norm_over": "row", "qk_norm_eps": self.norm_eps,
            "rotation": "neighbours", "chunk": int((sizes.get("mask") or {}).get("size", 0) or 0), "sink": True,
            "gate": "sigmoid_head", "position": position,
            "names": {"q_proj.weight": "q", "k_proj.weight": "k", "o_proj.weight": "o", "q_proj.bias": "q.b",
                      "k_proj.bias": "k.b", "o_proj.bias": "o.b", "q_norm.weight": "q.norm", "k_norm.weight": "k.norm",
                      "g_proj.weight": "g", "sink": "sink"},
        })

    def _schedule(self) -> list[int]:
        order = list(range(len(self.layers)))
        if not self.loop:
            return order
        start, stop, times = (int(self.loop[key]) for key in ("start", "stop", "times"))
        return order[:start] + order[start:stop] * times + order[stop:]

    def to_spec(self) -> ModelSpec:
        norm = PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "name": "", "add_scale": self.residual_mult})
        names = {"mixer_norm": "norm1", "mixer": "mix.", "feed_forward": "mlp."}
        layers = []
        for index, layer in enumerate(self.layers):
            mlp = layer.get("mlp")
            feed_forward = None if mlp is None else PartSpec("dense", {
                "hidden_size": self.width, "intermediate_size": int(mlp["ff"]), "activation": "relu_squared"})
            layers.append(LayerSpec(arrangement="shared_norm", mixer=self._mixer(layer), feed_forward=feed_forward,
                                    norm=norm, prefix=f"l{index}.", names=names))
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "name": "",
                                                   "scale": self.embedding_scale, "opens_stream": True}),
            layers=tuple(layers), schedule=tuple(ScheduleEntry(index) for index in self._schedule()), final_norm=norm,
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied": False, "name": ""}),
            final_norm_prefix="final.norm", embedding_prefix="embed", head_prefix="head",
        )
        spec.validate()
        return spec
