"""Small Vesidra configurations and seeded weights for the tests (test-side code only).

The configurations differ from one another in every size: head counts, plain, rotated and value sizes that differ from
each other, latents that are multiples of 16 (the tensor-core kernels), of 8 and of nothing, key rows that fit 64, 128 and
192 entries, rotations with and without YaRN scaling whose ramp covers all, some and none of the pairs, dense and routed
feed-forwards and none, with and without a shared expert. "ones" sets to 1 what can be 1. Weights are drawn so that every
tensor matters: norm gains away from 1, router biases that decide some choices, gates that do not saturate.
"""
from __future__ import annotations

import copy
import os

import numpy as np
import torch

import tiny_models as tm


def mla(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0, yarn=None):
    rot = {"base": base, "dims": rot_dim}
    if yarn is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim,
                                                  "kv_rank": kv_rank, "scale": scale, "rot": rot}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def _cfg(vocab, width, scale, eps, layers):
    return {"architecture": "Vesidra", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "layers": [dict(mixer, mlp=mlp) for mixer, mlp in layers]}


CONFIGS = {
    # key rows of 64 and 96 entries; a latent whose columns leave warps of the tensor-core kernel idle; a layer without
    # feed-forward; different rotations in different layers, with and without scaling
    "mixed": _cfg(203, 88, 6.5, 1e-5, [
        (mla(3, 40, 24, 36, 48, 0.15, 20000.0, (4.0, 60, 8.0, 1.0)), moe(7, 2, 40, shared=56)),
        (mla(2, 64, 32, 96, 80, 0.1, 500.0), dense(120)),
        (mla(5, 20, 16, 28, 112, 0.2, 1e6, (16.0, 4096, 32.0, 1.0)), None),
        (mla(2, 24, 8, 16, 24, 0.25, 10000.0, (2.5, 100, 4.0, 2.0)), moe(5, 4, 24)),
    ]),
    # sizes that are no multiple of 8 or of a warp
    "odd": _cfg(101, 50, 1.7, 1e-6, [
        (mla(3, 10, 6, 14, 22, 0.3, 1000.0, (3.0, 77, 5.0, 0.5)), dense(30)),
        (mla(5, 7, 2, 9, 11, 0.4, 10.0), moe(6, 3, 18, shared=10)),
    ]),
    # whatever can be 1 is 1: one head, one plain entry, a latent of one entry, one expert of which one is chosen, a scaling
    # by 1, an embedding scale of 1
    "ones": _cfg(64, 32, 1.0, 1e-3, [
        (mla(1, 1, 2, 1, 1, 1.0, 100.0, (1.0, 1, 1.0, 1.0)), moe(1, 1, 1, shared=1)),
        (mla(1, 16, 4, 8, 16, 0.5), dense(1)),
    ]),
    # sizes of the tensor cores: key rows of 160 entries beside values of 128, many heads, a latent of 256
    "wide": _cfg(310, 136, 11.0, 1e-5, [
        (mla(4, 112, 48, 128, 128, 0.08, 70000.0, (8.0, 256, 16.0, 1.0)), moe(12, 3, 64, shared=96)),
        (mla(18, 32, 32, 64, 64, 0.125, 10000.0), dense(200)),
        (mla(6, 64, 64, 64, 256, 0.09, 1e5, (40.0, 512, 32.0, 1.0)), moe(4, 1, 48)),
    ]),
}


def steady(cfg):
    """The configuration with routers that choose every expert: the weights still come from the logits, but no choice can
    fall the other way. A bfloat16 model's stream differs from the plain implementation's by about a hundredth, which moves
    a token's logits by as much, and one expert chosen otherwise is no rounding error. Whole models in bfloat16 are compared
    under these routers; the choice itself is compared in float32 whole models and, in both dtypes, on the parts alone,
    where the plain implementation reads the same input rows."""
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        mlp = layer.get("mlp")
        if mlp is not None and mlp["kind"] == "moe":
            mlp["router"]["top"] = mlp["router"]["experts"]
    return cfg


def tensor_shapes(cfg):
    W = cfg["width"]
    shapes = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, d, r, vd, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        shapes.update({p + "norm1": (W,), p + "mix.q": (H * (d + r), W), p + "mix.dkv": (rank + r, W), p + "mix.dkv.norm": (rank,),
                       p + "mix.uk": (H * d, rank), p + "mix.uv": (H * vd, rank), p + "mix.g": (H, W), p + "mix.o": (W, H * vd)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            shapes.update({p + "mlp.gate": (mlp["ff"], W), p + "mlp.up": (mlp["ff"], W), p + "mlp.down": (W, mlp["ff"])})
            continue
        F, n = mlp["expert"]["ff"], mlp["router"]["experts"]
        shapes.update({p + "mlp.router": (n, W), p + "mlp.router.b": (n,)})
        for e in range(n):
            shapes.update({f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
        if mlp.get("shared") is not None:
            S = mlp["shared"]["ff"]
            shapes.update({p + "mlp.shared.up": (S, W), p + "mlp.shared.down": (W, S)})
    return shapes


def bf16_exact(w):
    """float32 values that a bfloat16 file holds exactly (so both dtypes see one model)."""
    w = np.asarray(w, dtype=np.float32)
    return (tm.to_bf16_bits(w).astype(np.uint32) << 16).view(np.float32).reshape(w.shape)


def make_weights(cfg, seed):
    rng = np.random.Generator(np.random.PCG64(seed))
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        z = rng.standard_normal(shape).astype(np.float32)
        last = name.split(".")[-1]
        if last in ("norm1", "norm"):
            w = 1.0 + 0.2 * z
        elif name.endswith("router.b"):
            w = 0.5 * z
        elif last in ("router", "g"):
            w = 1.5 * z / np.sqrt(shape[-1])
        elif name == "embed":       # also the head: rows of a length that leaves the logits of the order of one
            w = z / np.sqrt(shape[-1])
        else:
            w = 1.2 * z / np.sqrt(shape[-1])
        out[name] = bf16_exact(w)
    return out


def write_folder(tmp, name, seed=0, bf16=False, cfg=None):
    cfg = cfg or CONFIGS[name]
    folder = os.path.join(str(tmp), f"vesidra_{name}")
    return tm.write_model_folder(folder, cfg, make_weights(cfg, seed), bf16=bf16)


def torch_weights(cfg, seed, dtype=torch.float64):
    return {k: torch.from_numpy(np.asarray(v)).to(dtype) for k, v in make_weights(cfg, seed).items()}


def prompts(cfg, lengths, seed=0):
    rng = np.random.Generator(np.random.PCG64(900 + seed))
    return [rng.integers(0, cfg["vocab"], size=n).tolist() for n in lengths]
