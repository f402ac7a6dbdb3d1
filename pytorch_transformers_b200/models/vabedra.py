"""Vabedra as an assembly of parts: VabedraConfig -> ModelSpec, with the checkpoint's tensor names.

Every layer is a ``post_norm`` block. Its mixer is a ``delta_rule`` with one decay per head and a full silu gate, or a
``normed_pair`` of a ``sink_attention`` (biases on q, k and v, normed and partly rotated queries and keys with frequencies
scaled by wavelength, soft-capped scores, a window that keeps the first tokens, one added to the softmax's denominator) and
a ``delta_rule`` with a decay per key channel and a sigmoid gate, both of low rank. The feed-forward is ``routed_experts``
with clamped units, scored by a softmax over all experts and chosen with a correction; a layer may have none. Each layer
ends with a ``gated_table`` token input from its columns of one table. The embeddings are scaled; the residual stream is
float32; the head is a tensor of its own. Tensor names: ``embed``, ``side.embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``
(``l<i>.mix.left.*``, ``l<i>.mix.right.*``), ``l<i>.mlp.*``, ``l<i>.side.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.vabedra import VabedraConfig
from ..parts.base import ModelSpec, PartSpec

GLU_ALPHA = 1.702       # g * sigmoid(1.702 g): fixed by the design
SINK_VALUE = 0.0        # one added to the softmax's denominator: a sink whose score is 0
PAIR_MULT = 0.5         # half the sum of the two normed branches


def _norm(cfg: VabedraConfig, name: str) -> PartSpec:
    return PartSpec("norm", "rmsnorm", {"size": cfg.width, "eps": float(cfg.norm["eps"])}, names={"weight": name})


def _delta(cfg: VabedraConfig, m: dict, p: str, channel: bool) -> PartSpec:
    own = ("a1", "a2", "g1", "g2") if channel else ("a", "g")
    names = {n: p + n for n in ("q", "k", "v", "b", "norm", "o", "dt_bias") + own}
    names.update({"a_log": p + "A_log"}, **{f"{n}_conv": f"{p}{n}.conv" for n in ("q", "k", "v")})
    kind = {"decay": "channel", "gate": "low_rank", "gate_act": "sigmoid"} if channel else {"decay": "head", "gate": "full", "gate_act": "silu"}
    return PartSpec("mixer", "delta_rule",
                    dict(kind, hidden=cfg.width, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"],
                         taps=m["conv"], eps=float(cfg.norm["eps"]), rank=m.get("rank")), names=names)


def _attention(cfg: VabedraConfig, m: dict, p: str) -> PartSpec:
    mask, rot = m.get("mask") or {}, m.get("rot") or {}
    children = {}
    if int(rot.get("dims", 0)) > 0:
        sc = rot.get("scaling")
        bands = {k: float(sc[k]) for k in ("factor", "low", "high", "original")} if sc else None
        children["position"] = PartSpec("position", "rotary", {"head_dim": m["dim"], "theta": float(rot["base"]),
                                                               "rotary_dim": int(rot["dims"]), "bands": bands})
    window = int(mask.get("size", 0))
    names = {n: p + n for n in ("q", "k", "v", "o")}
    names.update({f"{n}_b": f"{p}{n}.b" for n in ("q", "k", "v")}, q_norm=p + "q.norm", k_norm=p + "k.norm")
    return PartSpec("mixer", "sink_attention",
                    {"hidden": cfg.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
                     "scale": float(m["scale"]), "eps": float(cfg.norm["eps"]), "sink": False, "sink_value": SINK_VALUE,
                     "gate": False, "bias": True, "out_bias": False, "qk_norm": True, "qk_gain": True, "norm_first": True,
                     "softcap": float(m.get("softcap") or 0.0), "window": window,
                     "keep_first": int(mask.get("keep_first", 0)) if window > 0 else 0}, children=children, names=names)


def _mixer(cfg: VabedraConfig, i: int) -> PartSpec:
    m, p = cfg.layers[i]["mixer"], f"l{i}.mix."
    if cfg.layers[i]["type"] == "delta":
        return _delta(cfg, m, p, channel=False)
    return PartSpec("mixer", "normed_pair", {"hidden": cfg.width, "eps": float(cfg.norm["eps"]), "mult": PAIR_MULT},
                    children={"left": _attention(cfg, m["left"], p + "left."), "right": _delta(cfg, m["right"], p + "right.", channel=True)},
                    names={"left_out": p + "left.out", "right_out": p + "right.out"})


def _feed_forward(cfg: VabedraConfig, i: int) -> PartSpec:
    mlp, p = cfg.layers[i]["mlp"], f"l{i}.mlp."
    r = mlp["router"]
    names = {"router": p + "router", "correction": p + "correction"}
    names.update({f"e{e}.{t}": f"{p}e{e}.{t}" for e in range(r["experts"]) for t in ("gate", "up", "down")})
    return PartSpec("feed_forward", "routed_experts",
                    {"hidden": cfg.width, "inner": mlp["expert"]["ff"], "experts": r["experts"], "top": r["top"], "score": "softmax",
                     "correction": True, "expert": "clamped_glu", "limit": float(mlp["expert"]["limit"]), "alpha": GLU_ALPHA},
                    names=names)


def vabedra_block(cfg: VabedraConfig, i: int) -> PartSpec:
    children = {"mixer": _mixer(cfg, i), "norm_mixer": _norm(cfg, f"l{i}.norm1")}
    if cfg.layers[i].get("mlp") is not None:
        children.update(feed_forward=_feed_forward(cfg, i), norm_ff=_norm(cfg, f"l{i}.norm2"))
    if cfg.token_side is not None:
        dim = int(cfg.token_side["dim"])
        children["token_input"] = PartSpec("token_input", "gated_table",
                                           {"hidden": cfg.width, "dim": dim, "first": i * dim, "eps": float(cfg.norm["eps"])},
                                           names={n: f"l{i}.side.{n}" for n in ("gate", "proj", "norm")})
    return PartSpec("block", "post_norm", {"alpha": float(cfg.postln_alpha)}, children=children)


def vabedra_spec(cfg: VabedraConfig) -> ModelSpec:
    side = {}
    if cfg.token_side is not None:
        side = {"token_table_name": "side.embed", "token_table_width": len(cfg.layers) * int(cfg.token_side["dim"])}
    return ModelSpec(vocab_size=cfg.vocab, hidden_size=cfg.width, embedding_name="embed",
                     blocks=[vabedra_block(cfg, i) for i in range(len(cfg.layers))], final_norm=_norm(cfg, "final.norm"),
                     head_name="head", embedding_scale=float(cfg.embedding.get("scale", 1.0)), stream_float32=True, **side)
