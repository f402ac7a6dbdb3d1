"""A plain, slow restatement of the Vabedra design in float64, one function per mechanism, whole sequences at a time,
written from the design's equations. It shares no code with the package: the tests compare the two.

Notation: ``h`` [T, width] is a sublayer's input (the stream itself), weights are stored [out, in] and applied as ``W h``.
A model is (config dict as in config.json, dict of tensors by name).
"""
from __future__ import annotations

import math
from typing import Dict, List

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x ** 2).mean(dim=-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


# ---------------------------------------------------------------------------------------------- delta rule
def short_conv(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """y_t = sum_j taps[:, j] x_(t - n + 1 + j), zeros before the start; x [T, C], taps [C, n]."""
    T, n = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for j in range(n):
        back = n - 1 - j
        if back < T:
            y[back:] += taps[:, j] * x[:T - back]
    return y


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x ** 2).sum(dim=-1, keepdim=True) + 1e-6)


def delta_inputs(h, w: Dict[str, torch.Tensor], m: dict):
    """q, k [T, H, dim] (unit vectors, q scaled; every head's own copy), v [T, H, vdim], beta [T, H]."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = silu(short_conv(h @ w["q"].T, w["q.conv"])).reshape(T, G, d)
    k = silu(short_conv(h @ w["k"].T, w["k.conv"])).reshape(T, G, d)
    v = silu(short_conv(h @ w["v"].T, w["v.conv"])).reshape(T, H, dv)
    owner = torch.tensor([i // (H // G) for i in range(H)])
    return unit(q)[:, owner] * d ** -0.5, unit(k)[:, owner], v, sigmoid(h @ w["b"].T)


def delta_decay(h, w, m: dict) -> torch.Tensor:
    """g [T, H, dim]: one number per head, spread over its key channels, or one per head and key channel."""
    H, d = m["heads"], m["dim"]
    T = h.shape[0]
    if "a1" in w:
        z = (h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]
        sp = torch.log1p(torch.exp(-z.abs())) + z.clamp_min(0)
        return torch.exp(-torch.exp(w["A_log"])[None, :, None] * sp.reshape(T, H, d))
    z = h @ w["a"].T + w["dt_bias"]
    sp = torch.log1p(torch.exp(-z.abs())) + z.clamp_min(0)
    return torch.exp(-torch.exp(w["A_log"]) * sp)[:, :, None].expand(T, H, d)


def delta_recurrence(q, k, v, g, beta, state=None):
    """Per head: S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q. Returns (o [T, H, vdim], last S [H, dim, vdim])."""
    T, H, d = q.shape
    dv = v.shape[-1]
    S = torch.zeros(H, d, dv, dtype=q.dtype) if state is None else state.clone()
    o = torch.zeros(T, H, dv, dtype=q.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o, S


def delta_mixer(h, w, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    q, k, v, beta = delta_inputs(h, w, m)
    o, _ = delta_recurrence(q, k, v, delta_decay(h, w, m), beta)
    o = rms(o, eps) * w["norm"]
    gate = sigmoid((h @ w["g1"].T) @ w["g2"].T) if "g1" in w else silu(h @ w["g"].T)
    return (o.reshape(T, -1) * gate) @ w["o"].T


# ---------------------------------------------------------------------------------------------- attention
def frequencies(rot: dict) -> List[float]:
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            wave, orig = 2 * math.pi / f, float(sc["original"])
            if wave > orig / float(sc["low"]):
                f = f / float(sc["factor"])
            elif wave >= orig / float(sc["high"]):
                s = (orig / wave - float(sc["low"])) / (float(sc["high"]) - float(sc["low"]))
                f = (1 - s) * f / float(sc["factor"]) + s * f
        out.append(f)
    return out


def rotate(x: torch.Tensor, rot: dict, first_pos: int = 0) -> torch.Tensor:
    """x [T, heads, d]: entries i and i + dims / 2 of a head turn by position * frequency_i."""
    dims = int((rot or {}).get("dims", 0))
    if dims == 0:
        return x
    y = x.clone()
    pos = torch.arange(first_pos, first_pos + x.shape[0], dtype=F64)
    for i, f in enumerate(frequencies(rot)):
        c, s = torch.cos(pos * f)[:, None], torch.sin(pos * f)[:, None]
        u, v = x[..., i], x[..., i + dims // 2]
        y[..., i], y[..., i + dims // 2] = u * c - v * s, v * c + u * s
    return y


def visible(T: int, mask: dict) -> torch.Tensor:
    """[i, j]: j <= i and (i - j < size or j < keep_first); no window without a size."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    size, keep = int((mask or {}).get("size", 0)), int((mask or {}).get("keep_first", 0))
    return (j <= i) & (((i - j) < size) | (j < keep)) if size > 0 else j <= i


def sink_softmax(s: torch.Tensor, seen: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum exp(s_j)) over the keys that are seen."""
    s = s.masked_fill(~seen, -math.inf)
    top = s.max(dim=-1, keepdim=True).values.clamp_min(0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attention_mixer(h, w, m: dict, eps: float) -> torch.Tensor:
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = rotate(rms((h @ w["q"].T + w["q.b"]).reshape(T, H, d), eps) * w["q.norm"], m.get("rot"))
    k = rotate(rms((h @ w["k"].T + w["k.b"]).reshape(T, G, d), eps) * w["k.norm"], m.get("rot"))
    v = (h @ w["v"].T + w["v.b"]).reshape(T, G, dv)
    seen = visible(T, m.get("mask"))
    cap = float(m.get("softcap") or 0.0)
    out = []
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * float(m["scale"])
        if cap > 0:
            s = cap * torch.tanh(s / cap)
        out.append(sink_softmax(s, seen) @ v[:, g])
    return torch.cat(out, -1) @ w["o"].T


def parallel_mixer(h, w, m: dict, eps: float) -> torch.Tensor:
    left = attention_mixer(h, sub(w, "left."), m["left"], eps)
    right = delta_mixer(h, sub(w, "right."), m["right"], eps)
    return 0.5 * (rms(left, eps) * w["left.out"] + rms(right, eps) * w["right.out"])


# ---------------------------------------------------------------------------------------------- feed-forward
def expert(h, gate, up, down, limit: float) -> torch.Tensor:
    g = (h @ gate.T).clamp(max=limit)
    u = (h @ up.T).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ down.T


def route(h, w_router, correction, top: int):
    z = h @ w_router.T
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    ids = (s + correction).topk(top, -1).indices
    return ids, s.gather(1, ids)


def moe(h, w, mlp: dict) -> torch.Tensor:
    ids, weights = route(h, w["router"], w["correction"], int(mlp["router"]["top"]))
    out = torch.zeros(h.shape[0], w["e0.down"].shape[0], dtype=h.dtype)
    for e in range(int(mlp["router"]["experts"])):
        t, slot = (ids == e).nonzero(as_tuple=True)
        if len(t):
            out[t] += weights[t, slot][:, None] * expert(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"],
                                                         float(mlp["expert"]["limit"]))
    return out


# ---------------------------------------------------------------------------------------------- the model
def sub(weights: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(F64) for k, v in weights.items() if k.startswith(prefix)}


def token_side(x, e, w, eps: float) -> torch.Tensor:
    """x + the RMS-normed projection of gelu(gate x) * e, e the tokens' rows of this layer's part of the table."""
    return x + rms((gelu_tanh(x @ w["gate"].T) * e) @ w["proj"].T, eps) * w["norm"]


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens: List[int], streams: list = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence fed whole; ``streams`` (a list) receives the stream after every layer."""
    eps, alpha = float(config["norm"]["eps"]), float(config["postln_alpha"])
    ids = torch.tensor(tokens)
    x = weights["embed"].to(F64)[ids] * float(config["embedding"]["scale"])
    dim = int((config.get("token_side") or {}).get("dim", 0))
    for i, layer in enumerate(config["layers"]):
        mix = {"delta": delta_mixer, "parallel": parallel_mixer}[layer["type"]]
        x = rms(alpha * x + mix(x, sub(weights, f"l{i}.mix."), layer["mixer"], eps), eps) * weights[f"l{i}.norm1"].to(F64)
        if layer.get("mlp") is not None:
            x = rms(alpha * x + moe(x, sub(weights, f"l{i}.mlp."), layer["mlp"]), eps) * weights[f"l{i}.norm2"].to(F64)
        if dim:
            e = weights["side.embed"].to(F64)[ids, i * dim:(i + 1) * dim]
            x = token_side(x, e, sub(weights, f"l{i}.side."), eps)
        if streams is not None:
            streams.append(x.clone())
    return (rms(x, eps) * weights["final.norm"].to(F64)) @ weights["head"].to(F64).T
