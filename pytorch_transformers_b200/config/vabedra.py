"""Configuration of the Vabedra design: a decoder whose layers are listed one by one; the norms come after the sums, on a
stream that keeps ``postln_alpha`` times itself, and every layer takes an input of its own from the token ids. A layer's
mixer is a gated delta rule with one decay per head (``delta``), or an attention beside a gated delta rule with a decay per
key channel (``parallel``); its feed-forward is a mixture of experts with clamped units, or there is none.

config.json keys: ``architecture`` ("Vabedra"), ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``postln_alpha``,
``token_side.dim`` and ``layers``: a list of ``{"type", "mixer": {...}, "mlp": {...} | null}``. A ``delta`` mixer gives
``heads, kv_heads, dim, vdim, conv``; a ``parallel`` mixer ``right`` with the same keys and ``left``: ``heads, kv_heads, dim,
vdim, scale[, softcap][, mask: {size, keep_first}][, rot: {base, dims[, scaling: {factor, low, high, original}]}]``. The low
ranks of ``right`` are sizes of its tensors; ``right.rank`` names them for weights drawn at random. An ``mlp`` of kind ``moe``
gives ``expert: {ff, limit}`` and ``router: {experts, top}``.
"""
from __future__ import annotations

import dataclasses
from typing import Any, ClassVar, Dict, List, Optional

from .base import ModelConfig, _require
from .figudra import _whole
from .pafevik import _positive_int

MIXERS = ("delta", "parallel")


def _check_delta(m: Any, where: str) -> None:
    _require(isinstance(m, dict), f"{where} must be an object")
    for key in ("heads", "kv_heads", "dim", "vdim", "conv"):
        _positive_int(m.get(key), f"{where}.{key}")
    _require(m["heads"] % m["kv_heads"] == 0, f"{where}.heads must be a multiple of kv_heads")


def _check_attention(m: Any, where: str) -> None:
    _require(isinstance(m, dict), f"{where} must be an object")
    for key in ("heads", "kv_heads", "dim", "vdim"):
        _positive_int(m.get(key), f"{where}.{key}")
    _require(m["heads"] % m["kv_heads"] == 0, f"{where}.heads must be a multiple of kv_heads")
    _require(float(m.get("scale") or 0) > 0, f"{where}.scale must be positive")
    _require(float(m.get("softcap") or 0) >= 0, f"{where}.softcap must not be negative")
    mask = m.get("mask") or {}
    _require(isinstance(mask, dict), f"{where}.mask must be an object")
    size, keep = mask.get("size", 0), mask.get("keep_first", 0)
    _require(_whole(size) and size >= 0 and _whole(keep) and keep >= 0, f"{where}.mask.size and keep_first must be integers >= 0")
    rot = m.get("rot") or {}
    dims = rot.get("dims", 0)
    _require(_whole(dims) and 0 <= dims <= m["dim"] and dims % 2 == 0, f"{where}.rot.dims must be even and at most dim")
    _require(dims == 0 or float(rot.get("base", 0)) > 0, f"{where}.rot.base must be positive")
    sc = rot.get("scaling")
    _require(sc is None or (isinstance(sc, dict) and all(float(sc.get(k) or 0) > 0 for k in ("factor", "low", "high", "original"))),
             f"{where}.rot.scaling must give positive factor, low, high and original")


def _check_mlp(mlp: Any, where: str) -> None:
    _require(isinstance(mlp, dict) and mlp.get("kind") == "moe", f"{where}.kind must be 'moe'")
    _require(isinstance(mlp.get("expert"), dict), f"{where}.expert must be an object")
    _positive_int(mlp["expert"].get("ff"), f"{where}.expert.ff")
    _require(float(mlp["expert"].get("limit") or 0) > 0, f"{where}.expert.limit must be positive")
    r = mlp.get("router")
    _require(isinstance(r, dict), f"{where}.router must be an object")
    _positive_int(r.get("experts"), f"{where}.router.experts")
    _positive_int(r.get("top"), f"{where}.router.top")
    _require(r["top"] <= r["experts"], f"{where}.router.top must not exceed experts")


@dataclasses.dataclass
class VabedraConfig(ModelConfig):
    model_type: ClassVar[str] = "vabedra"

    architecture: str = "Vabedra"
    vocab: int = 0
    width: int = 0
    layers: List[Dict[str, Any]] = dataclasses.field(default_factory=list)
    norm: Dict[str, Any] = dataclasses.field(default_factory=lambda: {"eps": 1e-6})
    embedding: Dict[str, Any] = dataclasses.field(default_factory=lambda: {"scale": 1.0})
    postln_alpha: float = 1.0
    token_side: Optional[Dict[str, Any]] = None
    tie_word_embeddings: bool = False        # the head is a tensor of its own

    def __post_init__(self) -> None:
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        _require(isinstance(self.layers, list) and len(self.layers) > 0, "layers must be a non-empty list")
        _require(isinstance(self.norm, dict) and float(self.norm.get("eps", 0)) > 0, "norm.eps must be positive")
        _require(isinstance(self.embedding, dict) and isinstance(self.embedding.get("scale", 1.0), (int, float)),
                 "embedding.scale must be a number")
        _require(isinstance(self.postln_alpha, (int, float)), "postln_alpha must be a number")
        if self.token_side is not None:
            _require(isinstance(self.token_side, dict), "token_side must be an object")
            _positive_int(self.token_side.get("dim"), "token_side.dim")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            _require(isinstance(layer, dict) and layer.get("type") in MIXERS,
                     f"{where}.type must be one of {', '.join(MIXERS)}, got {layer.get('type') if isinstance(layer, dict) else layer!r}")
            m = layer.get("mixer")
            if layer["type"] == "delta":
                _check_delta(m, f"{where}.mixer")
            else:
                _require(isinstance(m, dict), f"{where}.mixer must be an object with left and right")
                _check_attention(m.get("left"), f"{where}.mixer.left")
                _check_delta(m.get("right"), f"{where}.mixer.right")
            if layer.get("mlp") is not None:
                _check_mlp(layer["mlp"], f"{where}.mlp")

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
