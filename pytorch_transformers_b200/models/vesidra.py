"""Vesidra as an assembly of parts: VesidraConfig -> ModelSpec, with the checkpoint's tensor names.

Every layer is a ``parallel`` block with one RMS norm whose output both the mixer and the feed-forward read. The mixer is a
``latent_attention`` with full-rank queries, one gate per head, and a rotation by halves with YaRN frequencies on the
shared key part. The feed-forward is a ``gated`` unit (silu) or ``routed_experts``: plain experts with the square of relu,
a biased router whose weights are the softmax over the chosen logits, and a ``dense`` shared expert of the same form; a
layer may have none. The embeddings are scaled as they enter the float32 residual stream; the head is the embedding table.
Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``.
"""
from __future__ import annotations

from ..config.vesidra import VesidraConfig
from ..parts.base import ModelSpec, PartSpec

EXPERT_ACTIVATION = "relu2"


def _norm(cfg: VesidraConfig, name: str) -> PartSpec:
    return PartSpec("norm", "rmsnorm", {"size": cfg.width, "eps": float(cfg.norm["eps"])}, names={"weight": name})


def _mixer(cfg: VesidraConfig, i: int) -> PartSpec:
    m, p = cfg.layers[i]["mixer"], f"l{i}.mix."
    rot = m["rot"]
    sc = rot.get("scaling")
    rotary = {"head_dim": m["rot_dim"], "rotary_dim": m["rot_dim"], "theta": float(rot["base"])}
    if sc is not None:
        rotary["yarn"] = {k: float(sc[k]) for k in ("factor", "original", "fast", "slow")}
    names = {n: p + n for n in ("q", "dkv", "uk", "uv", "g", "o")}
    names["dkv_norm"] = p + "dkv.norm"
    return PartSpec("mixer", "latent_attention",
                    {"hidden": cfg.width, "heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"], "vdim": m["vdim"],
                     "q_rank": None, "kv_rank": m["kv_rank"], "scale": float(m["scale"]), "eps": float(cfg.norm["eps"]),
                     "gate": "head", "wide_weights": True, "wide_out": True},
                    children={"position": PartSpec("position", "rotary", rotary)}, names=names)


def _feed_forward(cfg: VesidraConfig, i: int) -> PartSpec:
    mlp, p = cfg.layers[i]["mlp"], f"l{i}.mlp."
    if mlp["kind"] == "dense":
        return PartSpec("feed_forward", "gated", {"hidden": cfg.width, "inner": mlp["ff"], "activation": "silu", "wide_out": True},
                        names={n: p + n for n in ("gate", "up", "down")})
    r = mlp["router"]
    names = {"router": p + "router", "router_b": p + "router.b"}
    for e in range(r["experts"]):
        for t in ("up", "down"):
            names[f"e{e}.{t}"] = f"{p}e{e}.{t}"
    children = {}
    if mlp.get("shared") is not None:
        children["shared"] = PartSpec("feed_forward", "dense",
                                      {"hidden": cfg.width, "inner": mlp["shared"]["ff"], "activation": EXPERT_ACTIVATION,
                                       "wide_out": True},
                                      names={"up.weight": p + "shared.up", "down.weight": p + "shared.down"})
    return PartSpec("feed_forward", "routed_experts",
                    {"hidden": cfg.width, "inner": mlp["expert"]["ff"], "experts": r["experts"], "top": r["top"],
                     "score": "softmax_chosen", "correction": False, "router_bias": True, "expert": "plain",
                     "activation": EXPERT_ACTIVATION, "weight_on": "output"}, children=children, names=names)


def vesidra_block(cfg: VesidraConfig, i: int) -> PartSpec:
    children = {"norm_mixer": _norm(cfg, f"l{i}.norm1"), "mixer": _mixer(cfg, i)}
    if cfg.layers[i].get("mlp") is not None:
        children["feed_forward"] = _feed_forward(cfg, i)
    return PartSpec("block", "parallel", children=children)


def vesidra_spec(cfg: VesidraConfig) -> ModelSpec:
    return ModelSpec(vocab_size=cfg.vocab, hidden_size=cfg.width, embedding_name="embed",
                     blocks=[vesidra_block(cfg, i) for i in range(len(cfg.layers))], final_norm=_norm(cfg, "final.norm"),
                     head_name=None, embedding_scale=float(cfg.embedding.get("scale", 1.0)), stream_float32=True)
