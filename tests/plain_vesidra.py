"""A plain, slow restatement of the Vesidra design in float64, one function per mechanism, whole sequences at a
time, written from the design's equations. It shares no code with the package: the tests compare the two.

Notation: ``h`` [T, width] is what both sublayers of a layer read (the layer's normed stream), ``p`` a position (from
0), weights are stored [out, in] and applied as ``W h``. A model is (config dict as in config.json, dict of tensors by
name). Keys and values are written out per head: nothing is folded into the queries here.
"""
from __future__ import annotations

import math
from typing import Dict, List, Tuple

import torch

F64 = torch.float64


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last axis (eps inside the root), times a gain."""
    return x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z / (1.0 + torch.exp(-z))


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


# ---------------------------------------------------------------------------------------------- rotation
def frequencies(rot: dict) -> Tuple[List[float], float]:
    """(angle per position for every pair, the factor of the cosines and sines). Without ``scaling``: base^(-2i/dims)
    and 1. With it (YaRN): between the pairs that turn ``fast`` times or more within the ``original`` context, which
    keep their frequency, and those that turn ``slow`` times or fewer, whose frequency is divided by ``factor``,
    a linear ramp over the pair's index."""
    dims, base = int(rot["dims"]), float(rot["base"])
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return plain, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def index(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index(float(sc["fast"]))), 0)
    hi = min(math.ceil(index(float(sc["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(plain):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, ..., n]: entries i and i + dims/2 of the last axis are a pair, turned by position * frequency_i."""
    f, mult = frequencies(rot)
    half = len(f)
    out = x.clone()
    for i in range(half):
        a = positions.to(F64) * f[i]
        c, s = torch.cos(a) * mult, torch.sin(a) * mult
        while c.dim() < x.dim() - 1:
            c, s = c[:, None], s[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


# ---------------------------------------------------------------------------------------------- latent attention
def latent_rows(h, w: Dict[str, torch.Tensor], m: dict, eps: float, positions):
    """What a token leaves for later tokens: the normed latent [T, kv_rank] and the rotated key part [T, rot_dim]."""
    down = h @ w["dkv"].T
    return rms_norm(down[:, :m["kv_rank"]], w["dkv.norm"], eps), rotate(down[:, m["kv_rank"]:], positions, m["rot"])


def causal_softmax(scores: torch.Tensor, first_query: int = 0) -> torch.Tensor:
    """Softmax over the keys j <= i of scores [queries, keys]; query row r is at position first_query + r."""
    q, k = scores.shape
    seen = torch.arange(k)[None, :] <= (first_query + torch.arange(q))[:, None]
    e = torch.exp(scores.masked_fill(~seen, -math.inf) - scores.masked_fill(~seen, -math.inf).max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def latent_heads(q, c, kr, w, m: dict, first_query: int = 0) -> torch.Tensor:
    """Queries [Q, H, dim + rot_dim] (rotated already) on the rows c [K, kv_rank], kr [K, rot_dim]: [Q, H, vdim]."""
    H, d, vd, rank = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
    uk, uv = w["uk"].reshape(H, d, rank), w["uv"].reshape(H, vd, rank)
    out = []
    for hh in range(H):
        keys, values = c @ uk[hh].T, c @ uv[hh].T
        s = (q[:, hh, :d] @ keys.T + q[:, hh, d:] @ kr.T) * float(m["scale"])
        out.append(causal_softmax(s, first_query) @ values)
    return torch.stack(out, 1)


def latent_attention(h, w, m: dict, eps: float) -> torch.Tensor:
    T, H = h.shape[0], m["heads"]
    pos = torch.arange(T)
    q = (h @ w["q"].T).reshape(T, H, m["dim"] + m["rot_dim"])
    q = torch.cat([q[..., :m["dim"]], rotate(q[..., m["dim"]:], pos, m["rot"])], -1)
    c, kr = latent_rows(h, w, m, eps, pos)
    o = latent_heads(q, c, kr, w, m)
    gate = 1.0 / (1.0 + torch.exp(-(h @ w["g"].T)))          # one number per head
    return (o * gate[:, :, None]).reshape(T, H * m["vdim"]) @ w["o"].T


# ---------------------------------------------------------------------------------------------- feed-forwards
def dense_ff(h, w) -> torch.Tensor:
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def expert(h, up, down) -> torch.Tensor:
    return relu_squared(h @ up.T) @ down.T


def route(h, w_router, bias, top: int):
    """(ids [T, top], weights [T, top]): the largest logits, and a softmax over those alone."""
    z = h @ w_router.T + bias
    best, ids = z.topk(top, -1)
    e = torch.exp(best - best.max(-1, keepdim=True).values)
    return ids, e / e.sum(-1, keepdim=True)


def moe_ff(h, w, mlp: dict) -> torch.Tensor:
    ids, weights = route(h, w["router"], w["router.b"], int(mlp["router"]["top"]))
    out = torch.zeros(h.shape[0], w["e0.down"].shape[0], dtype=F64)
    for t in range(h.shape[0]):
        for e, g in zip(ids[t].tolist(), weights[t]):
            out[t] += g * expert(h[t:t + 1], w[f"e{e}.up"], w[f"e{e}.down"])[0]
    if mlp.get("shared"):
        out = out + expert(h, w["shared.up"], w["shared.down"])
    return out


def feed_forward(h, w, mlp: dict) -> torch.Tensor:
    return dense_ff(h, w) if mlp["kind"] == "dense" else moe_ff(h, w, mlp)


# ---------------------------------------------------------------------------------------------- the model
def sub(weights: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(F64) for k, v in weights.items() if k.startswith(prefix)}


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens: List[int], streams: list = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence fed whole; ``streams`` (a list) receives the stream after every layer."""
    eps = float(config["norm"]["eps"])
    table = weights["embed"].to(F64)
    x = table[torch.tensor(tokens)] * float(config["embedding"]["scale"])
    for i, layer in enumerate(config["layers"]):
        h = rms_norm(x, weights[f"l{i}.norm1"].to(F64), eps)
        y = latent_attention(h, sub(weights, f"l{i}.mix."), layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, sub(weights, f"l{i}.mlp."), layer["mlp"])
        x = x + y
        if streams is not None:
            streams.append(x.clone())
    return rms_norm(x, weights["final.norm"].to(F64), eps) @ table.T
