"""The gated delta rule: a linear recurrence whose state is corrected towards the value at the key that is written.

With ``h`` the mixer's input, ``kv_heads`` query/key heads of ``dim`` entries that the ``heads`` value heads of ``vdim``
entries share (head h reads query/key head h // (heads / kv_heads)):

    q, k, v = silu(conv(W h))            a causal filter of ``taps`` weights per channel, zeros before the sequence's start
    q, k <- x / sqrt(sum(x^2) + 1e-6) per head;  q <- q / sqrt(dim)
    beta = sigmoid(W_b h), one per head
    l = -exp(A_log) softplus(W_a h + dt_bias)                 ``decay="head"``: one logarithm of a decay per head
    l = -exp(A_log) softplus(W_a2 (W_a1 h) + dt_bias)         ``decay="channel"``: one per head and key channel, low rank
    S <- diag(exp(l)) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q          S = 0 before the first token
    out = W_o ( rmsnorm per head (o) * gain * act(gate) )     the gain [vdim] is shared by the heads; act: ``gate_act``
    gate = W_g h (``gate="full"``) or W_g2 (W_g1 h) (``gate="low_rank"``), or none (``gate="none"``)

Per sequence the mixer keeps the convolution's last taps - 1 inputs and S in the cache's state area (float32, zero when a
sequence starts) and needs no pages. Unit norms, beta, decays, state and the heads' norm are float32 whatever the model
dtype. All input projections, the low-rank ones' first matrices included, are one product; the second matrices of decay
and gate are one product too (block by block in one matrix, float32 sums). Prompts of 256 tokens or more run in chunks of
64 where the tensor-core kernels take the sizes, everything else token by token; the two differ by float32 rounding. The
low ranks are the first sizes of ``W_a1`` and ``W_g1``: given as ``rank``, or read from the checkpoint's tensors.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .base import BuildContext, ParamDecl, Part, PartSpec, StateNeed, register_part
from .linear import linear
from .recurrent import SCAN_CHUNK, RecurrenceChunks

LOW_RANK_MULTIPLE = 32      # the low-rank products' inner size is padded to what the weight-streaming kernel takes
WORD = 8                    # columns of a projection that start a section begin at whole 16-byte words


def _up(n: int, multiple: int) -> int:
    return (n + multiple - 1) // multiple * multiple


@register_part("mixer", "delta_rule")
class GatedDeltaRule(Part):
    graph_safe = True

    def __init__(self, build: BuildContext, spec: PartSpec, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int,
                 taps: int, eps: float = 1e-6, decay: str = "head", gate: str = "full", gate_act: str = "silu",
                 rank: Optional[int] = None):
        super().__init__(build, spec)
        self.hidden, self.heads, self.kv_heads = int(hidden), int(heads), int(kv_heads)
        self.dim, self.vdim, self.taps, self.eps = int(dim), int(vdim), int(taps), float(eps)
        k = build.kernels
        if decay not in ("head", "channel") or gate not in ("full", "low_rank", "none") or gate_act not in ("silu", "sigmoid"):
            raise ValueError(f"delta rule: decay is 'head' or 'channel', gate 'full', 'low_rank' or 'none' with 'silu' or "
                             f"'sigmoid', got {decay!r}, {gate!r}, {gate_act!r}")
        if self.kv_heads <= 0 or self.heads % self.kv_heads:
            raise ValueError(f"delta rule: heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
        if not (0 < self.dim <= k.DELTA_MAX_DIM and self.vdim > 0 and 1 <= self.taps <= k.DELTA_MAX_TAPS):
            raise ValueError(f"the delta rule's kernels take keys of 1 to {k.DELTA_MAX_DIM} entries and 1 to {k.DELTA_MAX_TAPS} "
                             f"taps, got {dim} and {taps}")
        if SCAN_CHUNK != k.DELTA_CHUNK:
            raise ValueError("the chunk planner and the chunked kernel disagree on the chunk's size")
        self.decay, self.gate, self.gate_act = decay, gate, gate_act
        self.rank = None if rank is None else int(rank)
        self.channels = 2 * self.kv_heads * self.dim + self.heads * self.vdim
        self.p_in = self.p_low = self.p_conv = self.p_a_log = self.p_dt_bias = self.p_norm = self.p_o = None
        # columns of the projection: q, k, v, then what the settings ask for
        at = self.channels
        self.g_off = at
        at += self.heads * self.vdim if gate == "full" else 0
        self.b_off = at
        at += self.heads
        self.a_off = at
        at += self.heads if decay == "head" else 0
        self.low_off = _up(at, WORD)
        self.low = 0                                        # columns of the low-rank section, known once weights are bound

    def param_decls(self) -> Dict[str, ParamDecl]:
        H, G, d, vd, C = self.heads, self.kv_heads, self.dim, self.vdim, self.taps
        r = -1 if self.rank is None else self.rank          # -1: whatever the checkpoint's tensor has
        decls = {"q": ParamDecl((G * d, self.hidden)), "k": ParamDecl((G * d, self.hidden)), "v": ParamDecl((H * vd, self.hidden)),
                 "q_conv": ParamDecl((G * d, C), role="vector", std=0.4), "k_conv": ParamDecl((G * d, C), role="vector", std=0.4),
                 "v_conv": ParamDecl((H * vd, C), role="vector", std=0.4), "b": ParamDecl((H, self.hidden)),
                 "a_log": ParamDecl((H,), role="vector", std=0.5), "norm": ParamDecl((vd,), role="vector", init="one_plus_normal", std=0.1),
                 "o": ParamDecl((self.hidden, H * vd))}
        if self.decay == "head":
            decls.update({"a": ParamDecl((H, self.hidden)), "dt_bias": ParamDecl((H,), role="vector", std=1.0)})
        else:
            decls.update({"a1": ParamDecl((r, self.hidden)), "a2": ParamDecl((H * d, r), std=0.2),
                          "dt_bias": ParamDecl((H * d,), role="vector", std=1.0)})
        if self.gate == "full":
            decls["g"] = ParamDecl((H * vd, self.hidden))
        elif self.gate == "low_rank":
            decls.update({"g1": ParamDecl((r, self.hidden)), "g2": ParamDecl((H * vd, r), std=0.2)})
        return decls

    def bind(self, t: Dict[str, torch.Tensor]) -> None:
        pairs = [(t[a], t[b]) for a, b in (("a1", "a2"), ("g1", "g2")) if a in t]
        for first, second in pairs:
            if first.shape[0] != second.shape[1]:
                raise ValueError(f"delta rule: a low-rank projection's two matrices do not fit ({list(first.shape)}, {list(second.shape)})")
        rows = [t["q"], t["k"], t["v"]] + [t[n] for n in ("g", "b", "a") if n in t]
        rows.append(t["q"].new_zeros(self.low_off - sum(w.shape[0] for w in rows), self.hidden))
        ranks = sum(first.shape[0] for first, _ in pairs)
        self.low = _up(ranks, LOW_RANK_MULTIPLE)
        rows += [first for first, _ in pairs] + [t["q"].new_zeros(self.low - ranks, self.hidden)]
        self.p_in = torch.cat(rows).contiguous()
        if pairs:       # the second matrices, each on its own columns of the low-rank section
            self.p_low = t["q"].new_zeros(sum(s.shape[0] for _, s in pairs), self.low)
            at_row = at_col = 0
            for first, second in pairs:
                self.p_low[at_row:at_row + second.shape[0], at_col:at_col + first.shape[0]] = second
                at_row, at_col = at_row + second.shape[0], at_col + first.shape[0]
        self.p_conv = torch.cat([t["q_conv"], t["k_conv"], t["v_conv"]]).t().contiguous()      # [taps, channels]
        self.p_a_log, self.p_dt_bias, self.p_o = t["a_log"], t["dt_bias"], t["o"]
        self.p_norm = t["norm"].repeat(self.heads).contiguous()                                # the one gain, once per head

    # ---- the projected protocol (parts/pair.py)
    def in_rows(self) -> int:
        return self.p_in.shape[0] if self.p_in is not None else self.low_off + self.low

    def out_columns(self) -> int:
        return self.heads * self.vdim

    def in_weight(self):
        return self.p_in

    def out_weight(self):
        return self.p_o

    def release_projections(self) -> None:
        self.p_in = self.p_o = None

    def cache_need(self):
        return None

    def state_need(self):
        return StateNeed(self.build.kernels.delta_state_floats(self.heads, self.kv_heads, self.dim, self.vdim, self.taps))

    def planner(self):
        return RecurrenceChunks()

    def forward_projected(self, proj, ctx, entry, out, out_scale: float = 1.0) -> None:
        """``proj`` [tokens, in_rows()] -> the normed and gated heads [tokens, heads * vdim] into ``out``."""
        if out_scale != 1.0:
            raise ValueError("delta rule: the heads take no output factor")
        k = self.build.kernels
        H, G, d, vd = self.heads, self.kv_heads, self.dim, self.vdim
        z = gate = None
        if self.p_low is not None:
            low = linear(k, proj[:, self.low_off:self.low_off + self.low], self.p_low, wide_out=True)
            if self.decay == "channel":
                z = low[:, :H * d]
            if self.gate == "low_rank":
                gate = low[:, low.shape[1] - H * vd:]
        if self.gate == "full":
            gate = proj[:, self.g_off:self.g_off + H * vd]
        state = ctx.state_of(entry, self.state_need().numel)
        slots, batch = ctx.dev["slots"], ctx.batch_c[0]
        act, inv, logd, beta = k.delta_prepare(proj, self.p_conv, state, slots, batch, self.p_a_log, self.p_dt_bias, H, G, d, vd,
                                               self.b_off, self.a_off, z, single_tokens=ctx.is_decode)
        plan, chunks = ctx.plan(RecurrenceChunks.plan_key), None
        if plan.facts["n_chunks"] and k.delta_chunks_take(act, d, vd):
            chunks = (plan.dev["chunk_seq"], plan.dev["chunk_q0"], plan.dev["seq_chunk0"], plan.facts["n_chunks"])
        o = k.delta_rule(act, inv, logd, beta, state, slots, batch, H, G, d, vd, self.taps, chunks)
        k.head_norm_gate(o, self.p_norm, gate, H, self.eps, proj.dtype, gate_act=self.gate_act, out=out)

    def forward(self, x, ctx, entry):
        """float32 [tokens, hidden]: the output product's sums, unrounded (a float32 norm or sum follows)."""
        k = self.build.kernels
        proj = linear(k, x, self.p_in)
        heads = torch.empty((x.shape[0], self.out_columns()), dtype=x.dtype, device=x.device)
        self.forward_projected(proj, ctx, entry, heads)
        return linear(k, heads, self.p_o, wide_out=True)
