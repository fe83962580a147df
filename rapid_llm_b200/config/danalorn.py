"""Configuration of the Danalorn decoder: a list of layers, each with an attention over a cached latent, a grouped-query
attention without rotation, or a gated linear attention, and a squared-relu feed-forward (or none).

``config.json`` gives ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``embedding.bigram`` (``buckets``,
``mul_prev``, ``mul_cur``) and ``layers``: one entry a layer, ``type`` names the mixer (``latent_attention``, ``attention``
or ``gla``), ``mixer`` its sizes and constants, ``mlp`` the feed-forward (``kind`` ``dense``) or ``null``.  Layer ``i``'s
tensors start with ``l<i>.``.  The rank of a ``gla`` mixer's decay product is not in the file: it is the first extent of the
tensor ``mix.a1``, so the configuration is read from a folder (:meth:`DanalornConfig.from_folder`) or given ``decay_rank``
per mixer.

What the parts are built from:

* the embedding is ``summed_embedding`` without a position row: the scaled token row + the token-pair row, opening the
  float32 stream (``token_embedding`` where there is no ``bigram``);
* every layer is the arrangement ``sandwich``: a norm in front of and behind each sublayer, all plain ``rmsnorm``;
* ``latent_attention`` -> ``latent_attention`` with a query latent, ``rotation="neighbours"`` over the whole rotated part,
  a window of ``mask.size`` positions (none: all) and a sink.  ``kv_from: j`` makes the layer read the rows layer ``j``
  cached: in the run order its entry names entry ``j`` as ``cache_from``, and layer ``j`` keeps as many positions as its
  widest reader needs;
* ``attention`` -> ``gqa_attention`` with biases, a norm per head, no rotation, the query temperature ``q_temp``, slopes
  ``2^(-8 (h + 1) / heads)`` times the distance off the scores, a fixed sink of score 0 and a sigmoid gate entry by entry;
* ``gla`` -> ``gated_linear``;
* ``dense`` -> ``dense`` with ``relu_squared``;
* the model ends in an RMS norm (``final.norm``) and an untied ``head``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Mapping

from .model_spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MAX_POSITIONS = 1 << 20     # nothing tabulated bounds a sequence; the engine's max_seq_len does

WANTED = {
    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale"),
    "attention": ("heads", "kv_heads", "dim", "vdim", "scale"),
    "gla": ("heads", "dim", "vdim", "tau", "decay_rank"),
}


def distance_slopes(heads: int) -> list[float]:
    """What a unit of distance takes off a score, per head: ``2^(-8 (h + 1) / heads)``."""
    return [2.0 ** (-8.0 * (head + 1) / heads) for head in range(heads)]


@dataclass
class DanalornConfig:
    architecture = "Danalorn"
    model_type = "danalorn"

    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    bigram: dict[str, int] | None
    layers: list[dict[str, Any]]
    raw: dict[str, Any] = field(default_factory=dict)

    # -------------------------------------------------------------- reading #
    @classmethod
    def from_folder(cls, model_dir, raw: Mapping[str, Any], overrides: Mapping[str, Any] | None = None) -> "DanalornConfig":
        """As :meth:`from_dict`, with every ``gla`` mixer's ``decay_rank`` read from the shape of its ``mix.a1``."""
        raw = copy.deepcopy(dict(raw))
        raw.update(copy.deepcopy(dict(overrides or {})))
        shapes = None
        for index, layer in enumerate(raw.get("layers") or []):
            if layer.get("type") != "gla" or "decay_rank" in (layer.get("mixer") or {}):
                continue
            if shapes is None:
                from ..weights.safetensors_io import tensor_shapes

                shapes = tensor_shapes(model_dir)
            name = f"l{index}.mix.a1"
            if name not in shapes:
                raise ValueError(f"layer {index}: the decay's rank is the first extent of {name!r}, which is missing")
            layer.setdefault("mixer", {})["decay_rank"] = int(shapes[name][0])
        return cls.from_dict(raw)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], overrides: Mapping[str, Any] | None = None) -> "DanalornConfig":
        raw = copy.deepcopy(dict(raw))
        raw.update(copy.deepcopy(dict(overrides or {})))
        for key in ("vocab", "width", "layers", "norm"):
            if key not in raw:
                raise ValueError(f"config.json of a Danalorn model lacks {key!r}")
        embedding = raw.get("embedding") or {}
        bigram = embedding.get("bigram")
        if bigram:
            bigram = {key: int(bigram[key]) for key in ("buckets", "mul_prev", "mul_cur")}
        config = cls(vocab=int(raw["vocab"]), width=int(raw["width"]), norm_eps=float(raw["norm"]["eps"]),
                     embedding_scale=float(embedding.get("scale", 1.0)), bigram=bigram or None,
                     layers=list(raw["layers"]), raw=raw)
        config.validate()
        return config

    def validate(self) -> None:
        if not self.layers:
            raise ValueError("a Danalorn model needs at least one layer")
        for index, layer in enumerate(self.layers):
            kind, mixer = layer.get("type"), layer.get("mixer") or {}
            if kind not in WANTED:
                raise ValueError(f"layer {index}: unknown mixer type {kind!r}")
            for key in WANTED[kind]:
                if key not in mixer:
                    raise ValueError(f"layer {index}: the {kind} mixer lacks {key!r}")
            if kind == "latent_attention":
                self._validate_latent(index, mixer)
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {index}: unknown feed-forward kind {mlp.get('kind')!r}")

    def _validate_latent(self, index: int, mixer: Mapping[str, Any]) -> None:
        rot_dim = int(mixer["rot_dim"])
        if rot_dim and "base" not in (mixer.get("rot") or {}):
            raise ValueError(f"layer {index}: a rotated part needs rot.base")
        if rot_dim and int(mixer["rot"].get("dims", rot_dim)) != rot_dim:
            raise ValueError(f"layer {index}: a latent-attention mixer rotates its whole rotated part: rot.dims must equal rot_dim")
        source = mixer.get("kv_from")
        if source is None:
            return
        source = int(source)
        if not 0 <= source < index or self.layers[source].get("type") != "latent_attention":
            raise ValueError(f"layer {index}: kv_from must name an earlier latent_attention layer, got {source}")
        theirs = self.layers[source]["mixer"]
        if theirs.get("kv_from") is not None:
            raise ValueError(f"layer {index}: layer {source} has no latent of its own")
        if (int(theirs["kv_rank"]), int(theirs["rot_dim"])) != (int(mixer["kv_rank"]), rot_dim) \
                or (rot_dim and float(theirs["rot"]["base"]) != float(mixer["rot"]["base"])):
            raise ValueError(f"layer {index}: kv_rank, rot_dim and rotation must equal layer {source}'s, whose rows it reads")

    def to_dict(self) -> dict[str, Any]:
        embedding: dict[str, Any] = {"scale": self.embedding_scale}
        if self.bigram:
            embedding["bigram"] = dict(self.bigram)
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps}, "embedding": embedding, "layers": copy.deepcopy(self.layers)}

    # ----------------------------------------------------------------- spec #
    @staticmethod
    def _window(sizes: Mapping[str, Any]) -> int:
        return int((sizes.get("mask") or {}).get("size", 0) or 0)

    def _source(self, index: int) -> int | None:
        layer = self.layers[index]
        source = layer["mixer"].get("kv_from") if layer["type"] == "latent_attention" else None
        return None if source is None else int(source)

    def _kept(self, index: int) -> int:
        """Positions layer ``index`` must keep cached: the widest window among itself and the layers that read its
        rows; 0 (everything) as soon as one of them has no window."""
        readers = [other for other in range(index + 1, len(self.layers)) if self._source(other) == index]
        windows = [self._window(self.layers[at]["mixer"]) for at in (index, *readers)]
        return 0 if 0 in windows else max(windows)

    def _mixer(self, index: int) -> PartSpec:
        kind, sizes = self.layers[index]["type"], self.layers[index]["mixer"]
        if kind == "gla":
            return PartSpec("gated_linear", {
                "hidden_size": self.width, "num_heads": int(sizes["heads"]), "key_dim": int(sizes["dim"]),
                "value_dim": int(sizes["vdim"]), "decay_rank": int(sizes["decay_rank"]), "tau": float(sizes["tau"]),
                "norm_eps": self.norm_eps})
        if kind == "latent_attention":
            rot = sizes.get("rot") or {}
            shares = self._source(index) is not None
            return PartSpec("latent_attention", {
                "hidden_size": self.width, "num_heads": int(sizes["heads"]), "head_dim": int(sizes["dim"]),
                "rot_dim": int(sizes["rot_dim"]), "value_dim": int(sizes["vdim"]), "kv_rank": int(sizes["kv_rank"]),
                "q_rank": int(sizes["q_rank"]), "scale": float(sizes["scale"]), "norm_eps": self.norm_eps,
                "rotation": "neighbours", "sink": True, "window": self._window(sizes), "shares_cache": shares,
                "cache_window": None if shares else self._kept(index),
                "position": PartSpec("rotary_frequencies", {
                    "rotary_dim": int(sizes["rot_dim"]), "theta": float(rot.get("base", 1.0)), "max_positions": MAX_POSITIONS})})
        warm = sizes.get("q_temp")
        return PartSpec("gqa_attention", {
            "hidden_size": self.width, "num_heads": int(sizes["heads"]), "num_kv_heads": int(sizes["kv_heads"]),
            "head_dim": int(sizes["dim"]), "value_dim": int(sizes["vdim"]), "scale": float(sizes["scale"]),
            "qkv_bias": True, "qk_norm": True, "qk_norm_eps": self.norm_eps, "gate": "sigmoid", "gate_rides": True,
            "slopes": distance_slopes(int(sizes["heads"])), "sink_score": 0.0,
            "temperature": None if not warm else (float(warm["coef"]), float(warm["every"])),
            "position": PartSpec("none", {"max_positions": MAX_POSITIONS}),
            "names": {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o",
                      "q_proj.bias": "q.b", "k_proj.bias": "k.b", "v_proj.bias": "v.b", "g_proj.weight": "g",
                      "q_norm.weight": "q.norm", "k_norm.weight": "k.norm"}})

    def _feed_forward(self, mlp: Mapping[str, Any] | None) -> PartSpec | None:
        if mlp is None:
            return None
        return PartSpec("dense", {"hidden_size": self.width, "intermediate_size": int(mlp["ff"]),
                                  "activation": "relu_squared"})

    def to_spec(self) -> ModelSpec:
        norm = PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "name": ""})
        layers = tuple(LayerSpec(arrangement="sandwich", mixer=self._mixer(index),
                                 feed_forward=self._feed_forward(layer.get("mlp")), norm=norm, prefix=f"l{index}.")
                       for index, layer in enumerate(self.layers))
        embedding = {"vocab_size": self.vocab, "hidden_size": self.width, "scale": self.embedding_scale, "name": "embed"}
        if self.bigram:
            embedding = PartSpec("summed_embedding", {
                **embedding, "pair_buckets": self.bigram["buckets"], "pair_mul_prev": self.bigram["mul_prev"],
                "pair_mul_cur": self.bigram["mul_cur"], "pair_name": "bigram"})
        else:
            embedding = PartSpec("token_embedding", {**embedding, "opens_stream": True})
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, max_positions=MAX_POSITIONS,
            embedding=embedding, layers=layers,
            schedule=tuple(ScheduleEntry(index, cache_from=self._source(index)) for index in range(len(self.layers))),
            final_norm=norm,
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied": False, "name": ""}),
            final_norm_prefix="final.norm", embedding_prefix="", head_prefix="head",
        )
        spec.validate()
        return spec
