"""Small Vabedra configurations and seeded weights for the tests (test-side code only).

The configurations differ from one another in every size: heads and shared heads, key and value sizes that differ from
each other and are no multiple of 8, filters of one to six taps, low ranks from 1 to 40, windows shorter than a page, longer
than a page and longer than any prompt, kept first tokens from none to more than a page, rotations over a part of a head,
over all of it and none, with and without frequencies scaled by wavelength (kept, mixed and divided ones), caps, clamps,
token inputs of several sizes and none, layers without a feed-forward and every order of the two mixers. "ones" sets to 1
what can be 1. Weights are drawn so that every tensor matters: gains away from 1, decays from nearly closed to nearly open,
router rows large enough that the choice differs from token to token and small enough that the scores stay apart.
"""
from __future__ import annotations

import copy
import os

import numpy as np
import torch

import tiny_models as tm


def delta(heads, kv_heads, dim, vdim, conv, rank=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}
    return m if rank is None else dict(m, rank=rank)


def att(heads, kv_heads, dim, vdim, scale, softcap=None, window=0, keep=0, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap is not None:
        m["softcap"] = softcap
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), rot[2:]))
    return m


def moe(experts, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def _cfg(vocab, width, eps, alpha, scale, side, layers):
    out = []
    for mixer, mlp in layers:
        kind = "parallel" if isinstance(mixer, tuple) else "delta"
        out.append({"type": kind, "mixer": {"left": mixer[0], "right": mixer[1]} if kind == "parallel" else mixer, "mlp": mlp})
    cfg = {"architecture": "Vabedra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
           "embedding": {"scale": scale}, "layers": out}
    if side:
        cfg["token_side"] = {"dim": side}
    return cfg


CONFIGS = {
    # both orders, a layer without feed-forward, shared key heads, windows shorter and longer than a page
    "mixed": _cfg(211, 96, 1e-5, 1.7, 3.0, 20, [
        (delta(4, 2, 24, 20, 4), moe(6, 2, 40, 0.7)),
        ((att(6, 2, 24, 20, 0.6, softcap=4.0, window=33, keep=5, rot=(8, 10000.0, 4.0, 1.0, 3.0, 64)), delta(3, 3, 16, 40, 3, rank=8)),
         moe(9, 3, 24, 1.5)),
        (delta(6, 3, 32, 16, 2), None),
        ((att(2, 1, 32, 32, 0.3, softcap=2.5, window=70, keep=0, rot=(32, 500.0)), delta(2, 1, 40, 24, 5, rank=12)), moe(4, 1, 56, 3.0)),
    ]),
    # sizes that are no multiple of 8 or of a warp; more kept tokens than a page holds; no token input; no cap
    "odd": _cfg(97, 52, 1e-6, 0.8, 1.0, 0, [
        ((att(5, 5, 10, 14, 0.4, window=129, keep=70, rot=(6, 10000.0, 2.0, 0.5, 8.0, 200)), delta(3, 1, 6, 10, 6, rank=5)), None),
        (delta(2, 1, 37, 11, 3), moe(5, 2, 18, 0.9)),
    ]),
    # whatever can be 1 is 1: one head, a window of one, one kept token, one expert, one tap, rank 1, one column a token input
    "ones": _cfg(64, 32, 1e-6, 1.0, 1.0, 1, [
        ((att(1, 1, 16, 16, 1.0 / 16, softcap=1.0, window=1, keep=1, rot=(2, 10.0)), delta(1, 1, 8, 8, 1, rank=1)), moe(1, 1, 16, 1.0)),
        (delta(1, 1, 8, 16, 1), moe(2, 1, 8, 1.0)),
    ]),
    # head sizes of the tensor cores; windows of 130 and longer than every prompt
    "wide": _cfg(300, 128, 1e-5, 2.2, 8.0, 33, [
        ((att(8, 2, 64, 64, 0.2, softcap=15.0, window=130, keep=4, rot=(32, 100000.0, 8.0, 1.0, 4.0, 100)), delta(4, 2, 64, 64, 4, rank=40)),
         moe(16, 4, 64, 2.0)),
        (delta(4, 1, 64, 128, 4), moe(8, 2, 48, 1.2)),
        ((att(4, 4, 128, 128, 0.1, softcap=30.0, window=1000, keep=6, rot=(64, 10000.0)), delta(2, 2, 128, 64, 3, rank=16)), None),
        (delta(2, 2, 128, 128, 2), moe(6, 3, 40, 0.8)),
    ]),
}


def steady(cfg):
    """The configuration with routers that choose every expert: the weights still come from the scores, but no choice can fall
    the other way. A bfloat16 model's stream differs from the plain implementation's by a rounding, which moves a token's
    scores; among a handful of scores some pair at the edge of the choice is that close now and then, the token then runs
    another expert, and the recurrent layers carry the difference on. Whole models in bfloat16 are compared under these
    routers; the choice itself is compared in float32 whole models and, in both dtypes, on the parts alone."""
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        if layer.get("mlp") is not None:
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return cfg


def delta_shapes(m, W, p, channel):
    H, G, d, vd, n = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    out = {"q": (G * d, W), "k": (G * d, W), "v": (H * vd, W), "q.conv": (G * d, n), "k.conv": (G * d, n), "v.conv": (H * vd, n),
           "b": (H, W), "A_log": (H,), "norm": (vd,), "o": (W, H * vd)}
    if channel:
        r = m["rank"]
        out.update({"a1": (r, W), "a2": (H * d, r), "dt_bias": (H * d,), "g1": (r, W), "g2": (H * vd, r)})
    else:
        out.update({"a": (H, W), "dt_bias": (H,), "g": (H * vd, W)})
    return {p + k: v for k, v in out.items()}


def attention_shapes(m, W, p):
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    out = {"q": (H * d, W), "q.b": (H * d,), "k": (G * d, W), "k.b": (G * d,), "v": (G * vd, W), "v.b": (G * vd,), "q.norm": (d,),
           "k.norm": (d,), "o": (W, H * vd)}
    return {p + k: v for k, v in out.items()}


def mixer_shapes(layer, W, p):
    if layer["type"] == "delta":
        return delta_shapes(layer["mixer"], W, p, False)
    return dict(attention_shapes(layer["mixer"]["left"], W, p + "left."), **delta_shapes(layer["mixer"]["right"], W, p + "right.", True),
                **{p + "left.out": (W,), p + "right.out": (W,)})


def tensor_shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    shapes = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    side = (cfg.get("token_side") or {}).get("dim", 0)
    if side:
        shapes["side.embed"] = (V, side * len(cfg["layers"]))
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        shapes[p + "norm1"] = (W,)
        shapes.update(mixer_shapes(layer, W, p + "mix."))
        if side:
            shapes.update({p + "side.gate": (side, W), p + "side.proj": (W, side), p + "side.norm": (W,)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        F, E = mlp["expert"]["ff"], mlp["router"]["experts"]
        shapes.update({p + "norm2": (W,), p + "mlp.router": (E, W), p + "mlp.correction": (E,)})
        for e in range(E):
            shapes.update({f"{p}mlp.e{e}.gate": (F, W), f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
    return shapes


def bf16_exact(w):
    """float32 values that a bfloat16 file holds exactly (so both dtypes see one model)."""
    w = np.asarray(w, dtype=np.float32)
    return (tm.to_bf16_bits(w).astype(np.uint32) << 16).view(np.float32).reshape(w.shape)


def draw(name, shape, rng):
    z = rng.standard_normal(shape).astype(np.float32)
    last = name.split(".")[-1]
    if last in ("norm1", "norm2", "norm", "out"):
        w = 1.0 + 0.2 * z
    elif last == "A_log":
        w = 0.7 * z
    elif last == "dt_bias":
        w = -1.0 + 2.0 * z              # decays from nearly closed to nearly open
    elif last == "conv":
        w = z / np.sqrt(shape[-1]) + (np.arange(shape[-1]) == shape[-1] - 1)
    elif last == "correction":
        w = 0.05 * z
    elif last == "b" and len(shape) == 1:
        w = 0.5 * z                     # the biases of q, k and v
    elif last in ("router", "a", "b", "a2"):
        w = 1.5 * z / np.sqrt(shape[-1])
    elif name in ("embed", "side.embed"):
        w = 0.7 * z
    else:
        w = 1.2 * z / np.sqrt(shape[-1])
    return bf16_exact(w)


def make_weights(cfg, seed):
    rng = np.random.Generator(np.random.PCG64(seed))
    return {name: draw(name, shape, rng) for name, shape in tensor_shapes(cfg).items()}


def write_folder(tmp, name, seed=0, bf16=False, cfg=None):
    cfg = cfg or CONFIGS[name]
    folder = os.path.join(str(tmp), f"vabedra_{name}")
    return tm.write_model_folder(folder, cfg, make_weights(cfg, seed), bf16=bf16)


def torch_weights(cfg, seed, dtype=torch.float64):
    return {k: torch.from_numpy(np.asarray(v)).to(dtype) for k, v in make_weights(cfg, seed).items()}


def prompts(cfg, lengths, seed=0):
    rng = np.random.Generator(np.random.PCG64(900 + seed))
    return [rng.integers(0, cfg["vocab"], size=n).tolist() for n in lengths]
