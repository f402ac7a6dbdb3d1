"""Configuration of the Vesidra design: a decoder whose layers are listed one by one. Every layer is a parallel block (one
RMS norm; the mixer and the feed-forward both read its output) around a latent attention: full-rank queries, keys and
values through one low-rank latent per token, a rotated key part that all heads share (YaRN-scaled frequencies, pairs
half the rotated size apart), one sigmoid gate per head. The feed-forward is a dense gated unit or a mixture of plain
experts (the square of relu) with a softmax over the chosen logits and a shared expert; a layer may have none. The
embeddings are scaled, and the head is the embedding table.

config.json keys: ``architecture`` ("Vesidra"), ``vocab``, ``width``, ``embedding.scale``, ``norm.eps`` and ``layers``: a
list of ``{"type": "latent_attention", "mixer": {...}, "mlp": {...} | null}``. A mixer gives ``heads, dim, rot_dim, vdim,
kv_rank, scale, rot: {base[, dims][, scaling: {factor, original, fast, slow}]}``; ``rot.dims`` is ``rot_dim``. An ``mlp`` of
kind ``dense`` gives ``ff``; of kind ``moe`` ``expert: {ff}``, ``router: {experts, top}`` and optionally ``shared: {ff}``.
"""
from __future__ import annotations

import dataclasses
from typing import Any, ClassVar, Dict, List

from .base import ModelConfig, _require
from .pafevik import _positive_int

MIXERS = ("latent_attention",)


def _positive(value: Any) -> bool:
    return isinstance(value, (int, float)) and not isinstance(value, bool) and value > 0


def _check_mixer(m: Any, where: str) -> None:
    _require(isinstance(m, dict), f"{where}.mixer must be an object")
    for key in ("heads", "dim", "rot_dim", "vdim", "kv_rank"):
        _positive_int(m.get(key), f"{where}.mixer.{key}")
    _require(m["rot_dim"] % 2 == 0, f"{where}.mixer.rot_dim must be even")
    _require(_positive(m.get("scale")), f"{where}.mixer.scale must be positive")
    rot = m.get("rot")
    _require(isinstance(rot, dict) and _positive(rot.get("base")), f"{where}.mixer.rot.base must be positive")
    _require(rot.get("dims", m["rot_dim"]) == m["rot_dim"], f"{where}.mixer.rot.dims must equal rot_dim")
    sc = rot.get("scaling")
    if sc is not None:
        _require(isinstance(sc, dict) and all(_positive(sc.get(k)) for k in ("factor", "original", "fast", "slow")),
                 f"{where}.mixer.rot.scaling must give positive factor, original, fast and slow")
        _require(rot["base"] != 1, f"{where}.mixer.rot.base must not be 1 beside a scaling")


def _check_mlp(mlp: Any, where: str) -> None:
    _require(isinstance(mlp, dict) and mlp.get("kind") in ("dense", "moe"), f"{where}.mlp.kind must be 'dense' or 'moe'")
    if mlp["kind"] == "dense":
        _positive_int(mlp.get("ff"), f"{where}.mlp.ff")
        return
    _require(isinstance(mlp.get("expert"), dict), f"{where}.mlp.expert must be an object")
    _positive_int(mlp["expert"].get("ff"), f"{where}.mlp.expert.ff")
    r = mlp.get("router")
    _require(isinstance(r, dict), f"{where}.mlp.router must be an object")
    _positive_int(r.get("experts"), f"{where}.mlp.router.experts")
    _positive_int(r.get("top"), f"{where}.mlp.router.top")
    _require(r["top"] <= r["experts"], f"{where}.mlp.router: cannot choose {r['top']} of {r['experts']} experts")
    if mlp.get("shared") is not None:
        _require(isinstance(mlp["shared"], dict), f"{where}.mlp.shared must be an object")
        _positive_int(mlp["shared"].get("ff"), f"{where}.mlp.shared.ff")


@dataclasses.dataclass
class VesidraConfig(ModelConfig):
    model_type: ClassVar[str] = "vesidra"

    architecture: str = "Vesidra"
    vocab: int = 0
    width: int = 0
    embedding: Dict[str, Any] = dataclasses.field(default_factory=lambda: {"scale": 1.0})
    layers: List[Dict[str, Any]] = dataclasses.field(default_factory=list)
    norm: Dict[str, Any] = dataclasses.field(default_factory=lambda: {"eps": 1e-6})
    tie_word_embeddings: bool = True         # the head is the embedding table, without its scale

    def __post_init__(self) -> None:
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        _require(isinstance(self.layers, list) and len(self.layers) > 0, "layers must be a non-empty list")
        _require(isinstance(self.norm, dict) and _positive(self.norm.get("eps")), "norm.eps must be positive")
        _require(isinstance(self.embedding, dict) and _positive(self.embedding.get("scale", 1.0)),
                 "embedding.scale must be positive")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            _require(isinstance(layer, dict) and layer.get("type") in MIXERS,
                     f"{where}.type must be one of {', '.join(MIXERS)}, got {layer.get('type') if isinstance(layer, dict) else layer!r}")
            _check_mixer(layer.get("mixer"), where)
            if layer.get("mlp") is not None:
                _check_mlp(layer["mlp"], where)

    # the names that the rest of the library uses for the sizes every decoder has
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)
