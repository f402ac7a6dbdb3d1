"""The latent-attention mixer: queries and keys/values both go through a low-rank latent, and only the
key/value latent (RMS-normed) and one rotated key part shared by all heads are cached per token.

With ``h`` the mixer's input, H heads, per head ``dim`` plain and ``rot_dim`` rotated query/key
entries, values of size ``vdim``, latent sizes ``q_rank`` and ``kv_rank``:

    c_q = rmsnorm(W_dq h) * w_qn        q = W_uq c_q      laid out per head as [dim plain | rot_dim to rotate]
    [c_raw | kr_raw] = W_dkv h          c = rmsnorm(c_raw) * w_kvn,   kr = rotate(kr_raw, position)
    k_h = W_uk[h] c,  v_h = W_uv[h] c
    score_h(i, j) = (q_plain_h(i) . k_h(j) + rotate(q_rot_h(i)) . kr(j)) * scale,   j <= i
    out = W_o (concat_h softmax(score_h) v_h  *  sigmoid(W_g h))

The cache row of a token is [c | kr] (one row for all heads, no value pool). The kernels use
``q_plain_h . (W_uk[h] c) = (W_uk[h]^T q_plain_h) . c``: the key up-projection is folded into the query,
every head scores against the cached rows themselves, and the softmax-weighted sum of the latents
goes through W_uv[h] afterwards. Long prompts of a bfloat16 model whose per-head sizes fit the tcgen05
prompt kernel (64 or 128, or keys of 192 beside values of 128) take the unfolded way instead: the cached latents of
the step's sequences go through [W_uk; W_uv] in one library product into per-head keys and values in scratch pools,
and that kernel runs on them. A layer built with ``own_kv=False`` has no W_dkv: its schedule
entry reads the cache entry that another latent-attention layer writes.

Variants, all by constructor parameters: ``q_rank=None`` has no query latent, ``q = W_q h``; the projections of h
(queries, key/value latent, gate) are then one product. ``gate="head"``: W_g has a row per head, and a head's whole
output is multiplied by its sigmoid. ``wide_weights``: in the tensor-core kernels of a bfloat16 model the softmax
weights meet the values as two bfloat16 terms (16 bits of mantissa). ``wide_out``: without a tensor to add, the output
product's float32 sums are returned unrounded. The pairs that are rotated and the frequencies are the ``position``
child's.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .attention import AttentionTiles
from .base import BuildContext, CacheNeed, ParamDecl, Part, PartSpec, register_part
from .linear import linear


UNFOLD_MAX_BYTES = 8 << 30      # most scratch (per-head keys and values of every page) that the unfolded prompt path may hold


class LatentContext:
    """For prompts that the unfolded path takes: (sequence, position) of every cached row that the step's
    sequences will hold after it, in the order of the sequences. Steps of few tokens get an empty plan."""
    plan_key = "latent_context"

    def __init__(self, kernels):
        self.kernels = kernels

    def plan(self, ctx):
        from ..engine.batch import StepPlan
        if max(ctx.new) <= self.kernels.TC_TILE_TOKENS // 2:      # the tile lists hold 128 tokens a tile only beyond this
            return StepPlan(arrays={}, facts={"n_ctx": 0})
        seqs, poss = [], []
        for b, (p, n) in enumerate(zip(ctx.past, ctx.new)):
            seqs += [b] * (p + n)
            poss += range(p + n)
        return StepPlan(arrays={"ctx_seq": seqs, "ctx_pos": poss}, facts={"n_ctx": len(seqs)})


@register_part("mixer", "latent_attention")
class LatentAttention(Part):
    graph_safe = True
    fuses_add = True

    def __init__(self, build: BuildContext, spec: PartSpec, hidden: int, heads: int, dim: int, rot_dim: int, vdim: int,
                 q_rank: Optional[int], kv_rank: int, scale: float, eps: float, own_kv: bool = True, gate: str = "entry",
                 wide_weights: bool = False, wide_out: bool = False):
        super().__init__(build, spec)
        self.hidden, self.heads, self.dim, self.rot_dim, self.vdim = int(hidden), int(heads), int(dim), int(rot_dim), int(vdim)
        self.kv_rank, self.scale, self.eps, self.own_kv = int(kv_rank), float(scale), float(eps), bool(own_kv)
        self.q_rank = None if q_rank is None else int(q_rank)
        if gate not in ("entry", "head"):
            raise ValueError(f"the output gate is one per 'entry' or one per 'head', got {gate!r}")
        self.gate_per_head, self.wide_weights, self.wide_out = gate == "head", bool(wide_weights), bool(wide_out)
        self.gate_cols = self.heads * (1 if self.gate_per_head else int(vdim))
        if min(self.heads, self.dim, self.vdim, self.kv_rank) <= 0 or self.rot_dim < 0 or (self.q_rank is not None and self.q_rank <= 0):
            raise ValueError("latent attention needs positive head count, sizes and ranks")
        if self.kv_rank > 512:
            raise ValueError(f"the latent attention kernel keeps a row's sums in registers up to kv_rank 512, got {self.kv_rank}")
        self.position = self.children.get("position")
        self.interleaved = bool(getattr(self.position, "interleaved", False))
        self.p_dq = self.p_dq_norm = self.p_uq = self.p_side = self.p_dkv_norm = self.p_uk_t = self.p_uv = self.p_o = None
        self.p_ukv = self.p_in = None

    def param_decls(self) -> Dict[str, ParamDecl]:
        H = self.heads
        if self.q_rank is None:
            d = {"q": ParamDecl((H * (self.dim + self.rot_dim), self.hidden))}
        else:
            d = {"dq": ParamDecl((self.q_rank, self.hidden)),
                 "dq_norm": ParamDecl((self.q_rank,), role="vector", init="one_plus_normal"),
                 "uq": ParamDecl((H * (self.dim + self.rot_dim), self.q_rank))}
        d.update({"uk": ParamDecl((H * self.dim, self.kv_rank)),
                  "uv": ParamDecl((H * self.vdim, self.kv_rank)),
                  "g": ParamDecl((self.gate_cols, self.hidden)),
                  "o": ParamDecl((self.hidden, H * self.vdim))})
        if self.own_kv:
            d["dkv"] = ParamDecl((self.kv_rank + self.rot_dim, self.hidden))
            d["dkv_norm"] = ParamDecl((self.kv_rank,), role="vector", init="one_plus_normal")
        return d

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        H = self.heads
        self.p_o = tensors["o"]
        if self.q_rank is None:
            # all projections of h in one product; zero rows at the end bring the rows of the result to whole 16-byte words
            rows = [tensors["q"]] + ([tensors["dkv"]] if self.own_kv else []) + [tensors["g"]]
            spare = -sum(t.shape[0] for t in rows) % 8
            if spare:
                rows.append(tensors["q"].new_zeros((spare, self.hidden)))
            self.p_in = torch.cat(rows).contiguous()
        else:
            self.p_dq, self.p_dq_norm, self.p_uq = tensors["dq"], tensors["dq_norm"], tensors["uq"]
            # the gate and the key/value down-projection read the same input: one product
            self.p_side = torch.cat([tensors["g"], tensors["dkv"]]) if self.own_kv else tensors["g"]
        self.p_dkv_norm = tensors.get("dkv_norm")
        # W_uk per head, transposed: [H, kv_rank, dim] maps a head's plain query part into latent space
        self.p_uk_t = tensors["uk"].view(H, self.dim, self.kv_rank).transpose(1, 2).contiguous()
        self.p_uv = tensors["uv"].view(H, self.vdim, self.kv_rank)
        # for prompts through the unfolded path: keys and values of all heads from one product
        self.p_ukv = torch.cat([tensors["uk"], tensors["uv"]]) if self._unfold_size() else None

    def cache_need(self):
        return CacheNeed("full", 1, self.kv_rank + self.rot_dim, 0, v_head_dim=0) if self.own_kv else None

    def state_need(self):
        return None

    def planner(self):
        return [AttentionTiles(self.build.kernels), LatentContext(self.build.kernels)]

    def runs_beside(self, ctx) -> bool:
        """On a second stream while the cache rows that this layer reads in the step are few beside the feed-forward's
        weights (the limits are the kernels': kernels.decode_attention_fits_beside)."""
        if self.build.dtype != torch.bfloat16:
            return False
        row = self.kv_rank + self.rot_dim
        return self.build.kernels.decode_attention_fits_beside(sum(p + n for p, n in zip(ctx.past, ctx.new)) * row * 2, row)

    def _unfold_size(self):
        """Sizes (key row, value row) of the tcgen05 prompt kernel that hold this layer's keys and values, or None."""
        k = self.build.kernels
        if self.build.dtype != torch.bfloat16:
            return None
        for hd, hd_v in ((64, 64), (128, 128), (192, 128)):
            if self.dim + self.rot_dim <= hd and self.vdim <= hd_v and k.attention_tc_supports(hd, hd_v):
                return hd, hd_v
        return None

    def _unfold_pools(self, cache, group, hd, hd_v):
        """Scratch pools for the unfolded keys and values, laid out like the group's pages; kept on the cache.
        Layers of equal sizes share them (a layer rewrites every row that it reads)."""
        pages = cache.groups[group].k.shape[1]
        key = (group, self.heads, hd, hd_v, self.dim, self.rot_dim, self.vdim)
        pools = cache.__dict__.setdefault("_latent_unfold", {})
        if key not in pools:
            if pages * self.heads * 64 * (hd + hd_v) * 2 > UNFOLD_MAX_BYTES:
                pools[key] = None
            else:
                shape = (pages, self.heads, 64)     # zeroed: what lies beyond a head's entries must stay zero
                pools[key] = (torch.zeros(shape + (hd,), dtype=torch.bfloat16, device=self.build.device),
                              torch.zeros(shape + (hd_v,), dtype=torch.bfloat16, device=self.build.device))
        return pools[key]

    def _splits(self, ctx) -> int:
        """Blocks that share the key pages of a (token, 16 heads) tile in a step of single tokens: up to
        two blocks an SM, each with a page at least (8 sequences of 2,048 rows: 24 blocks 22.8 us, 33 blocks 21.6)."""
        k = self.build.kernels
        blocks = ctx.n_seqs * ((self.heads + k.LATENT_ROWS - 1) // k.LATENT_ROWS)
        return max(1, min((2 * k.sm_count(self.build.device)) // blocks, ctx.pages_hint, 128))

    def forward(self, x, ctx, entry, add=None):
        k = self.build.kernels
        t, H = x.shape[0], self.heads
        row = self.kv_rank + self.rot_dim
        if self.q_rank is None:
            proj, q_cols = linear(k, x, self.p_in), H * (self.dim + self.rot_dim)
            q = proj[:, :q_cols].view(t, H, self.dim + self.rot_dim)
            down, gate = proj[:, q_cols:q_cols + row], proj[:, q_cols + (row if self.own_kv else 0):][:, :self.gate_cols]
        else:
            cq = k.norm(linear(k, x, self.p_dq), self.p_dq_norm, None, self.eps, "rmsnorm")
            q = linear(k, cq, self.p_uq).view(t, H, self.dim + self.rot_dim)
            side = linear(k, x, self.p_side)
            gate, down = side[:, :self.gate_cols], side[:, self.gate_cols:]
        pool, _, group = ctx.cache.entry_storage(entry.cache_entry)
        batch = ctx.batch_c[group]
        rope = ctx.rope(self.position)
        if entry.writes_cache:
            if not self.own_kv:
                raise ValueError("a latent attention layer without a key/value projection cannot write a cache entry")
            k.latent_store(down, self.p_dkv_norm, self.eps, pool, batch, rope, self.kv_rank,
                           self.rot_dim, self.interleaved)
        tiles = ctx.plan(AttentionTiles.plan_key)
        rows = ctx.plan(LatentContext.plan_key)
        sizes = self._unfold_size()
        if sizes and rows.facts["n_ctx"] and tiles.facts["mma_tokens"] == k.TC_TILE_TOKENS:
            pools = self._unfold_pools(ctx.cache, group, *sizes)
            if pools is not None:
                # long prompts in bfloat16: per-head keys and values unfolded from the cached latents, and the
                # tcgen05 prompt kernel on them
                o = k.latent_unfolded_attention(q, pool, pools[0], pools[1], self.p_ukv, gate, batch, rows.dev["ctx_seq"],
                                                rows.dev["ctx_pos"], rows.facts["n_ctx"], tiles.dev["mtile_seq"],
                                                tiles.dev["mtile_q0"], tiles.facts["n_mma_tiles"], rope, self.dim,
                                                self.rot_dim, self.vdim, self.kv_rank, self.scale, self.interleaved,
                                                gate_per_head=self.gate_per_head, wide_weights=self.wide_weights)
                return self._out(o, add)
        q_abs = k.block_linear(q[:, :, :self.dim], self.p_uk_t, out_dtype=torch.float32)
        if tiles.facts["mma_tokens"] == 1:     # a step of single tokens: a tile is one token's heads
            o_lat = k.latent_attention(q_abs, q, self.dim, pool, batch, tiles.dev["mtile_seq"], tiles.dev["mtile_q0"],
                                       tiles.facts["n_mma_tiles"], 1, rope, self.kv_rank, self.rot_dim, self.scale,
                                       self.interleaved, n_splits=self._splits(ctx), wide_weights=self.wide_weights)
        else:
            o_lat = k.latent_attention(q_abs, q, self.dim, pool, batch, tiles.dev["tile_seq"], tiles.dev["tile_q0"],
                                       tiles.facts["n_tiles"], k.generic_tile_rows(), rope, self.kv_rank, self.rot_dim,
                                       self.scale, self.interleaved, wide_weights=self.wide_weights)
        o = k.block_linear(o_lat, self.p_uv, gate=gate, gate_per_group=self.gate_per_head)    # values up, times sigmoid(gate)
        return self._out(o.view(t, H * self.vdim), add)

    def _out(self, o, add):
        if add is None:
            return linear(self.build.kernels, o, self.p_o, wide_out=self.wide_out)
        return linear(self.build.kernels, o, self.p_o, add=add)
