"""Vesidra on the GPU against the plain implementation (tests/plain_vesidra.py), in float32 and bfloat16.

First every mechanism alone: the cached rows (latent norm, rotation with scaled frequencies), the output gate per head in
each of the kernels that apply it, the tensor-core attentions with key and value rows of different sizes and with the softmax
weights as two bfloat16 terms (rows whose values cancel show a rounded weight), the latent attention as a part (whole, in
portions, token by token, two sequences, a slot that is used again; one key that a query is aligned with, through the latent
or through the rotated part, far back and at page borders, in prompts and in single tokens), the router against the plain
one, the feed-forwards. Then whole models of several shapes: each request alone, the stream after every layer, a prompt and
then single tokens, portions down to two tokens, batches of unequal requests on a small cache whose slots and pages are used
again, long decoding through replayed graphs, both branches of a step on two streams and on one, greedy generation through
``generate`` and from the command line, and the trace runner as a child process.
"""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_vesidra as plain
import vesidra_models as vm

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]
F64 = torch.float64


def K():
    from pytorch_transformers_b200 import kernels
    return kernels


def tdtype(name):
    return getattr(torch, name)


def row_errors(got, ref):
    got, ref = got.double().cpu().reshape(-1, got.shape[-1]), ref.double().cpu().reshape(-1, ref.shape[-1])
    return (got - ref).norm(dim=1) / ref.norm(dim=1).clamp_min(1e-30)


def close(got, ref, dtype, what="", f32=1e-4, bf16=3e-2):
    """float32: every row within rounding of float32 sums and the rows' median well within. bfloat16: the rows' median
    within a bfloat16 model's rounding and 9 rows in 10 within twice that."""
    e = row_errors(got, ref)
    if dtype == "float32":
        assert e.max() < f32 and e.median() < f32 / 10, f"{what}: worst row error {e.max():.3g}, median {e.median():.3g}"
    else:
        assert e.median() < bf16 and (e < 2 * bf16).double().mean() >= 0.9, \
            f"{what}: median row error {e.median():.3g}, worst {e.max():.3g}"


def bf16_exact(t):
    return t.bfloat16().double()


class Mixer:
    """A mixer part alone on a cache of its own, fed rows directly."""

    def __init__(self, spec, weights, dtype):
        from pytorch_transformers_b200.parts.base import BuildContext, make_part
        self.k, self.dt = K(), tdtype(dtype)
        self.part = make_part(BuildContext(torch.device("cuda"), self.dt, self.k), spec)
        decls = self.part.param_decls()
        self.part.bind({n: weights[self.part.spec.names[n]].to(device="cuda", dtype=torch.float32 if d.role == "vector" else self.dt)
                        for n, d in decls.items()})
        self.planners = list(self.part.planner())

    def cache(self, max_tokens, max_slots=None):
        from pytorch_transformers_b200.cache.paged import Cache
        return Cache([(0, self.part.cache_need(), self.part.state_need())], max_tokens, self.dt, "cuda", max_slots=max_slots)

    def step(self, cache, slots, rows):
        from pytorch_transformers_b200.engine.batch import StepContext
        from pytorch_transformers_b200.parts.base import ScheduleEntry
        ctx = StepContext(cache, slots, [[0] * r.shape[0] for r in rows], 1, [[] for _ in rows], self.planners)
        x = torch.cat(rows).to(self.dt).cuda().contiguous()
        y = self.part.forward(x, ctx, ScheduleEntry(0, 0))
        assert y.dtype == torch.float32         # the output product's sums, unrounded
        ctx.commit()
        return list(y.double().cpu().split([r.shape[0] for r in rows]))

    def run_cut(self, cache, rows, cuts):
        """One sequence fed in portions of the given sizes; returns all its output rows."""
        s, at, got = cache.open(), 0, []
        for n in cuts:
            got.append(self.step(cache, [s], [rows[at:at + n]])[0])
            at += n
        cache.close(s)
        return torch.cat(got)


def spec_of(layer, width, eps=1e-5):
    """The mixer's and the feed-forward's specs of a one-layer configuration, with names that start at mix. and mlp."""
    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200.models.vesidra import vesidra_block
    cfg = ptb.VesidraConfig.from_dict({"vocab": 8, "width": width, "norm": {"eps": eps}, "layers": [layer]})
    block = vesidra_block(cfg, 0)

    def rename(s):
        s.names = {a: b[3:] for a, b in s.names.items()}
        for c in s.children.values():
            rename(c)
    for c in block.children.values():
        rename(c)
    return block.children["mixer"], block.children.get("feed_forward")


def layer_weights(layer, width, seed):
    cfg = {"vocab": 8, "width": width, "layers": [layer]}
    return {k[3:]: torch.from_numpy(v) for k, v in vm.make_weights(cfg, seed).items() if k.startswith("l0.")}


# ------------------------------------------------------------------------------------------------ small kernels
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,groups,n,kk", [(1, 3, 20, 24), (9, 18, 64, 32), (70, 5, 14, 10), (300, 4, 40, 24)])
def test_values_up_with_a_gate_per_group(dtype, m, groups, n, kk):
    """Few rows (a warp per output), tens, and enough for the library's batched product: each with its epilogue."""
    k, dt = K(), tdtype(dtype)
    g = torch.Generator().manual_seed(m)
    x = torch.randn(m, groups, kk, generator=g).to(dt)
    w = (torch.randn(groups, n, kk, generator=g) / math.sqrt(kk)).to(dt)
    gate = (2 * torch.randn(m, 3 + groups + 5, generator=g)).to(dt)      # a stretch of wider rows
    got = k.block_linear(x.cuda(), w.cuda(), gate=gate.cuda()[:, 3:3 + groups], gate_per_group=True)
    want = torch.einsum("tgk,gnk->tgn", x.double(), w.double()) * torch.sigmoid(gate[:, 3:3 + groups].double())[:, :, None]
    close(got, want, dtype, "gate per group", f32=2e-6, bf16=5e-3)
    with pytest.raises(k.KernelError):
        k.block_linear(x.cuda(), w.cuda(), gate=gate.cuda()[:, :groups + 1], gate_per_group=True)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rank,rot,yarn", [(48, 24, (4.0, 60, 8.0, 1.0)), (22, 6, (3.0, 77, 5.0, 0.5)), (1, 2, (1.0, 1, 1.0, 1.0)),
                                           (80, 32, None), (512, 64, (40.0, 4096, 32.0, 1.0))])
def test_cached_rows(dtype, rank, rot, yarn):
    """The row a token leaves: its normed latent, and the key part rotated by its position with scaled frequencies."""
    m = vm.mla(2, 8, rot, 8, rank, 1.0, 20000.0, yarn)["mixer"]
    mixer_spec, _ = spec_of({"type": "latent_attention", "mixer": m}, 40)
    w = layer_weights({"type": "latent_attention", "mixer": m}, 40, rank)
    mixer = Mixer(mixer_spec, w, dtype)
    g = torch.Generator().manual_seed(rank)
    x = bf16_exact(torch.randn(150, 40, generator=g)).float()
    cache = mixer.cache(192)
    s, at = cache.open(), 0
    for n in (63, 2, 1, 84):
        mixer.step(cache, [s], [x[at:at + n]])
        at += n
    pool, _, gi = cache.entry_storage(0)
    rows = pool[torch.tensor(cache.pages(s, gi), device="cuda").long()].reshape(-1, rank + rot)[:150].double().cpu()
    c, kr = plain.latent_rows(x.double(), plain.sub(w, "mix."), m, 1e-5, torch.arange(150))
    if rank > 1:        # (a latent of one entry is its sign, and a float32 or bfloat16 sum near 0 may fall on either side)
        close(rows[:, :rank], c, dtype, "latent", f32=2e-5, bf16=1e-2)
    close(rows[:, rank:], kr, dtype, "rotated part", f32=2e-4, bf16=1e-2)


def _page_rows(cache, slot, pool, gi, n, values):
    """Write ``values`` [n, heads, entries] as the first n cached rows of a sequence."""
    pages = cache.pages(slot, gi)
    for p, page in enumerate(pages):
        part = values[p * 64:min(n, p * 64 + 64)]
        pool[page, :, :part.shape[0]] = part.transpose(0, 1).to(pool.dtype).cuda()


def _cancelling_values(p, v_dim, g):
    """Values [n, v_dim] under which the weighted sum nearly vanishes for the weights ``p`` [n]: neighbours' contributions are
    each other's negative up to the values' own bfloat16 rounding. What is left of the sum is as small as what a rounding of
    the weights to bfloat16 would do to it."""
    n = p.shape[0] // 2 * 2
    v = torch.zeros(p.shape[0], v_dim, dtype=F64)
    u = torch.randn(n // 2, v_dim, generator=g, dtype=F64)
    v[0:n:2] = u * p[1:n:2, None] / p.max()
    v[1:n:2] = -u * p[0:n:2, None] / p.max()
    return bf16_exact(v)


@pytest.mark.parametrize("dk,dv", [(64, 64), (128, 128), (192, 128)])
def test_prompt_attention_sizes_and_weights_in_two_terms(dk, dv):
    """The tcgen05 prompt attention with a key and a value head of its own per query head: against the plain softmax over
    one, several and very many pages, ragged tiles, two sequences, a prompt that goes on from a cache; and one row whose
    values cancel, where weights rounded to bfloat16 leave a large error and weights of two terms do not."""
    from pytorch_transformers_b200.cache.paged import Cache
    from pytorch_transformers_b200.engine.batch import StepContext
    from pytorch_transformers_b200.parts.attention import AttentionTiles
    from pytorch_transformers_b200.parts.base import CacheNeed
    k, dt, H = K(), torch.bfloat16, 3
    g = torch.Generator().manual_seed(dk)
    scale = 1.5 / math.sqrt(dk)
    for pasts, news in [((0,), (65,)), ((0, 0), (130, 200)), ((1, 500), (129, 70)), ((700,), (300,))]:
        totals = [p + n for p, n in zip(pasts, news)]
        cache = Cache([(0, CacheNeed("full", H, dk, 0, v_head_dim=dv), None)], sum((t + 63) // 64 * 64 for t in totals), dt, "cuda")
        slots = [cache.open() for _ in totals]
        for s, p in zip(slots, pasts):
            if p:
                cache.reserve_all([(s, p)])
                cache.commit(s, p)
        ctx = StepContext(cache, slots, [[0] * n for n in news], 1, [[] for _ in news], [AttentionTiles(k)])
        k_pool, v_pool, gi = cache.entry_storage(0)
        ks = [bf16_exact(torch.randn(t, H, dk, generator=g)) for t in totals]
        vs = [bf16_exact(torch.randn(t, H, dv, generator=g)) for t in totals]
        qs = [bf16_exact(torch.randn(t, H, dk, generator=g)) for t in news]
        weights = [[plain.causal_softmax(q[:, h] @ kk[:, h].T * scale, p) for h in range(H)] for q, kk, p in zip(qs, ks, pasts)]
        for b, t in enumerate(totals):
            vs[b][:, 1] = _cancelling_values(weights[b][1][-1], dv, g)       # head 1, the last row of every sequence
            _page_rows(cache, slots[b], k_pool, gi, t, ks[b])
            _page_rows(cache, slots[b], v_pool, gi, t, vs[b])
        want = [torch.stack([weights[b][h] @ vs[b][:, h] for h in range(H)], 1) for b in range(len(totals))]
        tiles = ctx.plan(AttentionTiles.plan_key)
        assert tiles.facts["mma_tokens"] == k.TC_TILE_TOKENS
        q = torch.cat(qs).to(dt).cuda().contiguous()
        args = (q, k_pool, v_pool, ctx.batch_c[gi], tiles.dev["mtile_seq"], tiles.dev["mtile_q0"], tiles.facts["n_mma_tiles"], H, scale)
        narrow, wide = (k.attention_tc(*args, wide_weights=w).double().cpu().view(-1, H, dv) for w in (False, True))
        k.check_device_errors("cuda")
        ref = torch.cat(want)
        for got in (narrow, wide):
            for h in (0, 2):
                assert row_errors(got[:, h], ref[:, h]).max() < 1e-2, f"{pasts} {news} head {h}"
        last = [sum(news[:b + 1]) - 1 for b in range(len(news))]
        assert row_errors(wide[last, 1], ref[last, 1]).max() < 0.03, f"{pasts} {news}"
        assert row_errors(narrow[last, 1], ref[last, 1]).min() > 0.1     # so the row does show the difference


@pytest.mark.parametrize("tokens,splits", [(1, 1), (1, 3), (16, 1)])
@pytest.mark.parametrize("rank,rot,heads", [(16, 0, 1), (48, 16, 3), (112, 32, 18), (256, 64, 20), (512, 64, 16)])
def test_latent_kernel_weights_in_two_terms(rank, rot, heads, tokens, splits):
    """Rows whose values cancel, in the tensor-core kernel of the folded form: entry 0 of the latent makes the scores, the
    other entries are values. Also latents whose columns do not divide among four warps."""
    from pytorch_transformers_b200.cache.paged import Cache
    from pytorch_transformers_b200.engine.batch import StepContext
    from pytorch_transformers_b200.parts.attention import AttentionTiles
    from pytorch_transformers_b200.parts.base import CacheNeed
    k, dt = K(), torch.bfloat16
    g = torch.Generator().manual_seed(rank + tokens)
    n, dk = 300, rank + rot
    assert k.latent_attention_mma_supports(rank, rot)
    cache = Cache([(0, CacheNeed("full", 1, dk, 0, v_head_dim=0), None)], 320, dt, "cuda")
    s = cache.open()
    cache.reserve_all([(s, n - tokens)])
    cache.commit(s, n - tokens)
    ctx = StepContext(cache, [s], [[0] * tokens], 1, [[]], [AttentionTiles(k)])
    pool, _, gi = cache.entry_storage(0)
    rows = torch.zeros(n, dk, dtype=F64)
    rows[:, 0] = bf16_exact(torch.randn(n, generator=g, dtype=F64))
    q_abs = torch.zeros(tokens, heads, rank, dtype=F64)
    q_abs[..., 0] = 1.0
    weights = plain.causal_softmax(rows[:, :1].T.expand(tokens, n) * 1.5, n - tokens)
    rows[:, 1:rank] = _cancelling_values(weights[-1], rank - 1, g)
    _page_rows(cache, s, pool, gi, n, rows[:, None])
    q = torch.zeros(tokens, heads, 4 + rot, dtype=dt, device="cuda")
    tiles = ctx.plan(AttentionTiles.plan_key)
    names = ("mtile_seq", "mtile_q0") if tokens == 1 else ("tile_seq", "tile_q0")
    args = (q_abs.float().cuda(), q, 4, pool, ctx.batch_c[gi], tiles.dev[names[0]], tiles.dev[names[1]], 1, tokens, None, rank, rot, 1.5)
    wide, narrow = (k.latent_attention(*args, n_splits=splits, wide_weights=w).double().cpu() for w in (True, False))
    ref = (weights @ rows[:, :rank])[:, None, :].expand(tokens, heads, rank)
    assert row_errors(wide[..., :1], ref[..., :1]).max() < 2e-2
    assert row_errors(wide[-1, :, 1:], ref[-1, :, 1:]).max() < 0.03
    assert row_errors(narrow[-1, :, 1:], ref[-1, :, 1:]).min() > 0.1
    assert row_errors(narrow[..., :1], ref[..., :1]).max() < 2e-2


# ------------------------------------------------------------------------------------------------ the mixer
MIXERS = [vm.mla(3, 40, 24, 36, 48, 0.15, 20000.0, (4.0, 60, 8.0, 1.0)),        # folded kernel: general; key rows of 64
          vm.mla(2, 64, 32, 96, 80, 0.1, 500.0),                               # tensor cores, five groups of columns; 128
          vm.mla(4, 112, 48, 128, 128, 0.08, 70000.0, (8.0, 256, 16.0, 1.0)),  # key rows of 160 in 192
          vm.mla(18, 32, 32, 64, 64, 0.125),                                   # more heads than a tile of one token has rows
          vm.mla(5, 7, 2, 9, 11, 0.4, 10.0), vm.mla(3, 10, 6, 14, 22, 0.3, 1000.0, (3.0, 77, 5.0, 0.5)),
          vm.mla(2, 150, 60, 40, 16, 0.08), vm.mla(1, 24, 16, 140, 32, 0.2),      # beyond the prompt kernel's sizes
          vm.mla(1, 16, 4, 8, 16, 0.5)]


def _id(layer):
    m = layer["mixer"]
    return f"{m['heads']}h{m['dim']}+{m['rot_dim']}x{m['vdim']}r{m['kv_rank']}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", MIXERS, ids=_id)
def test_latent_attention_whole_in_portions_and_single_tokens(layer, dtype):
    width = 40
    w = layer_weights(layer, width, layer["mixer"]["dim"])
    mixer = Mixer(spec_of(layer, width)[0], w, dtype)
    g = torch.Generator().manual_seed(2)
    x = bf16_exact(torch.randn(300, width, generator=g)).float()
    ref = plain.latent_attention(x.double(), plain.sub(w, "mix."), layer["mixer"], 1e-5)
    cache = mixer.cache(320, max_slots=1)
    for cuts in ([300], [130, 170], [64, 2, 3, 17, 214], [60] + [1] * 10 + [230], [1] * 70 + [230], [127, 1, 1, 171]):
        close(mixer.run_cut(cache, x, cuts), ref, dtype, f"cuts {cuts[:6]}", f32=2e-5, bf16=1.5e-2)
        cache.check()
    K().check_device_errors("cuda")
    y = bf16_exact(torch.randn(170, width, generator=g)).float()
    ref_y = plain.latent_attention(y.double(), plain.sub(w, "mix."), layer["mixer"], 1e-5)
    cache = mixer.cache(64 * 5)
    for heads in ((100, 62), (2, 130)):
        a, b = cache.open(), cache.open()
        out = mixer.step(cache, [a, b], [x[:heads[0]], y[:heads[1]]])
        got_x, got_y = [out[0]], [out[1]]
        for t in range(8):
            out = mixer.step(cache, [a, b], [x[heads[0] + t:heads[0] + t + 1], y[heads[1] + t:heads[1] + t + 1]])
            got_x.append(out[0]); got_y.append(out[1])
        close(torch.cat(got_x), ref[:heads[0] + 8], dtype, "first of two", f32=2e-5, bf16=1.5e-2)
        close(torch.cat(got_y), ref_y[:heads[1] + 8], dtype, "second of two", f32=2e-5, bf16=1.5e-2)
        cache.close(b); cache.close(a)      # the next pair finds slots and pages in another order


def copying_layer(heads, rank, rot_dim, base, yarn, scale):
    """A layer and weights under which a mixer's input row is (rotated query part | plain query part, shared by all heads |
    latent | rotated key part): the test writes queries, latents and key parts directly. Plain keys and values are the normed
    latent itself, every gate is open (sigmoid(0) = 1/2 of the value), the output projection is the identity."""
    layer = vm.mla(heads, rank, rot_dim, rank, rank, scale, base, yarn)
    width = 2 * (rank + rot_dim)
    q = torch.zeros(heads, rank + rot_dim, width)
    q[:, :, :rank + rot_dim] = torch.eye(rank + rot_dim)
    dkv = torch.zeros(rank + rot_dim, width)
    dkv[:, rank + rot_dim:] = torch.eye(rank + rot_dim)
    eye = torch.eye(rank).repeat(heads, 1)
    return layer, width, {"mix.q": q.reshape(-1, width), "mix.dkv": dkv, "mix.dkv.norm": torch.ones(rank), "mix.uk": eye,
                          "mix.uv": eye, "mix.g": torch.zeros(heads, width), "mix.o": torch.eye(heads * rank)}


NEEDLES = [(900, 3), (900, 0), (300, 63), (300, 64), (257, 255), (130, 127), (129, 128), (65, 64), (64, 63), (3, 1), (2, 0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("through", ["latent", "rotated"])
@pytest.mark.parametrize("rank,rot_dim", [(32, 16), (22, 8), (96, 32), (112, 64)])
def test_one_key_far_back_and_at_page_borders(rank, rot_dim, through, dtype):
    """The last query is aligned with one key among hundreds, through its latent or through the rotated part (the query is
    turned back by the distance, so that only the right scaled angles meet): that key's value answers."""
    layer, width, w = copying_layer(2, rank, rot_dim, 3000.0, (6.0, 120, 10.0, 1.0), 0.5)
    m = layer["mixer"]
    mixer = Mixer(spec_of(layer, width)[0], w, dtype)
    cache = mixer.cache(960)
    for n, at in NEEDLES:
        g = torch.Generator().manual_seed(n + at)
        x = torch.randn(n, width, generator=g)
        x[:, :rank + rot_dim] *= 0.2            # small queries: only the last one looks for something
        x[n - 1, :rank + rot_dim] = 0.0
        if through == "latent":
            d = torch.randn(rank, generator=g)
            x[at, rank + rot_dim:rank + rot_dim + rank] = d
            x[n - 1, :rank] = 24.0 * d / d.norm()
        else:
            d = torch.randn(rot_dim, generator=g)
            d = d / d.norm()
            x[at, -rot_dim:] = 9.0 * d          # other key parts have a norm of sqrt(rot_dim)
            back = plain.rotate(d[None].double(), torch.tensor([at - (n - 1)]), m["rot"])[0] / plain.frequencies(m["rot"])[1]
            x[n - 1, rank:rank + rot_dim] = 9.0 * back.float()
        x = bf16_exact(x).float()
        ref = plain.latent_attention(x.double(), plain.sub(w, "mix."), m, 1e-5)
        value = 0.5 * plain.rms_norm(x[at, rank + rot_dim:2 * rank + rot_dim].double(), torch.ones(rank), 1e-5)
        for cuts in ([n], [n - 1, 1], [max(1, n - 70)] + [min(70, n - 1)], [max(1, n - 20)] + [1] * min(20, n - 1)):
            got = mixer.run_cut(cache, x, cuts)
            close(got, ref, dtype, f"{n} tokens, key at {at}, cuts {cuts[:3]}", f32=5e-5)
            for h in range(2):
                assert (got[-1, h * rank:(h + 1) * rank] - value).norm() < 0.05 * value.norm(), f"{n} tokens, key at {at}, cuts {cuts[:3]}"
    K().check_device_errors("cuda")


def test_an_earlier_sequences_rows_are_not_seen_again():
    """Slots and pages that a longer sequence used: the next one must not see its keys, however strongly they answer."""
    layer, width, w = copying_layer(2, 32, 16, 1000.0, None, 1.0)
    mixer = Mixer(spec_of(layer, width)[0], w, "float32")
    cache = mixer.cache(128, max_slots=1)
    g = torch.Generator().manual_seed(0)
    x = torch.randn(128, width, generator=g) * 4
    mixer.run_cut(cache, x, [100, 28])
    y = torch.randn(70, width, generator=g)
    y[:, :32] = x[:70, 48:80]              # queries along the first sequence's latents
    ref = plain.latent_attention(y.double(), plain.sub(w, "mix."), layer["mixer"], 1e-5)
    for cuts in ([70], [5, 60, 5], [60] + [1] * 10):
        close(mixer.run_cut(cache, y, cuts), ref, "float32", f"cuts {cuts[:3]}", f32=2e-5)


# ------------------------------------------------------------------------------------------------ the feed-forwards
@pytest.mark.parametrize("n,top", [(1, 1), (5, 2), (8, 8), (33, 4), (64, 6), (256, 8)])
def test_router_against_the_plain_one(n, top):
    k = K()
    g = torch.Generator().manual_seed(n)
    for tokens in (1, 7, 700):
        h, wr, b = torch.randn(tokens, 24, generator=g), torch.randn(n, 24, generator=g), 2 * torch.randn(n, generator=g)
        ids, weights = plain.route(h.double(), wr.double(), b.double(), top)
        got_ids, got_w = k.route(h.cuda(), wr.cuda(), None, 1, 1, top, 1.0, "softmax_chosen", bias=b.cuda())
        got_ids = got_ids.cpu().long()
        # a choice may differ where two logits are within float32 rounding of each other
        same = (got_ids.sort(1).values == ids.sort(1).values).all(1)
        assert same.double().mean() > 0.99
        rows = same.nonzero().flatten()
        order = got_ids[rows].argsort(1)
        torch.testing.assert_close(got_w.double().cpu()[rows].gather(1, order), weights[rows].gather(1, ids[rows].argsort(1)),
                                   atol=1e-6, rtol=1e-5)
        torch.testing.assert_close(got_w.double().cpu().sum(1), torch.ones(tokens, dtype=F64), atol=1e-6, rtol=0)


def test_router_chooses_by_logits_also_where_a_softmax_over_all_would_vanish():
    """Logits 100 and more below the largest: exp(z - max) is 0 in float32 for all but one, the choice must not be by it.
    A correction moves the choice and not the weights; groups and a scale apply as for the other scores."""
    k = K()
    wr = torch.zeros(6, 8)
    b = torch.tensor([-300.0, 200.0, -110.0, -100.0, -400.0, -90.0])
    h = torch.zeros(3, 8)
    ids, w = k.route(h.cuda(), wr.cuda(), None, 1, 1, 3, 1.0, "softmax_chosen", bias=b.cuda())
    assert ids.cpu().tolist() == [[1, 5, 3]] * 3 and w.cpu().tolist() == [[1.0, 0.0, 0.0]] * 3
    corr = torch.tensor([0.0, -1000.0, 0.0, 0.0, 0.0, 0.0])
    ids, w = k.route(h.cuda(), wr.cuda(), corr.cuda(), 1, 1, 2, 2.0, "softmax_chosen", bias=b.cuda())
    assert ids.cpu().tolist() == [[5, 3]] * 3
    torch.testing.assert_close(w.double().cpu(), 2.0 * torch.softmax(torch.tensor([[-90.0, -100.0]] * 3, dtype=F64), 1), atol=1e-9, rtol=1e-5)
    ids, _ = k.route(h.cuda(), wr.cuda(), None, 3, 1, 2, 1.0, "softmax_chosen", bias=b.cuda())
    assert ids.cpu().tolist() == [[1, 0]] * 3           # the best group of two neighbours


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp,width", [(vm.dense(120), 88), (vm.dense(30), 50), (vm.dense(1), 32), (vm.moe(7, 2, 40, shared=56), 88),
                                       (vm.moe(6, 3, 18, shared=10), 50), (vm.moe(1, 1, 1, shared=1), 32), (vm.moe(5, 4, 24), 88),
                                       (vm.moe(40, 6, 64, shared=128), 128)])
def test_feed_forwards_against_the_plain_ones(mlp, width, dtype):
    from pytorch_transformers_b200.parts.base import BuildContext, make_part
    layer = dict(vm.mla(1, 8, 2, 8, 8, 1.0), mlp=mlp)
    w = layer_weights(layer, width, width)
    dt = tdtype(dtype)
    part = make_part(BuildContext(torch.device("cuda"), dt, K()), spec_of(layer, width)[1])
    for p in part.walk():
        decls = p.param_decls()
        p.bind({n: w[p.spec.names[n]].to(device="cuda", dtype=torch.float32 if d.role == "vector" else dt) for n, d in decls.items()})
    g = torch.Generator().manual_seed(5)
    for tokens in (1, 9, 300):
        h = bf16_exact(torch.randn(tokens, width, generator=g)).float()
        got = part.forward(h.to(dt).cuda(), None)
        assert got.dtype == torch.float32
        want = plain.feed_forward(h.double(), plain.sub(w, "mlp."), mlp)
        close(got, want, dtype, f"{mlp['kind']} {tokens} tokens", f32=2e-5)
        base = torch.randn(tokens, width, generator=g)
        close(part.forward(h.to(dt).cuda(), None, add=base.cuda()), want + base.double(), dtype, "with the stream", f32=2e-5)


# ------------------------------------------------------------------------------------------------ whole models
class Loaded:
    def __init__(self, tmp, name, dtype):
        import pytorch_transformers_b200 as ptb
        # bfloat16 models run routers that choose every expert (vesidra_models.steady says why)
        self.cfg = vm.CONFIGS[name] if dtype == "float32" else vm.steady(vm.CONFIGS[name])
        self.folder = vm.write_folder(tmp, name, seed=len(name), bf16=(dtype == "bfloat16"), cfg=self.cfg)
        self.model = ptb.AutoModelForCausalLM.from_pretrained(self.folder, dtype=dtype)
        self.w = vm.torch_weights(self.cfg, len(name))
        self._ref = {}

    def plain_logits(self, ids):
        key = tuple(ids)
        if key not in self._ref:
            self._ref[key] = plain.forward(self.cfg, self.w, ids)
        return self._ref[key]


@pytest.fixture(scope="module")
def loaded(tmp_path_factory):
    made = {}

    def get(name, dtype):
        if (name, dtype) not in made:
            made[(name, dtype)] = Loaded(tmp_path_factory.mktemp(f"{name}_{dtype}"), name, dtype)
        return made[(name, dtype)]
    return get


NAMES = sorted(vm.CONFIGS)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_each_request_alone_and_whole(loaded, name, dtype):
    L = loaded(name, dtype)
    assert L.model.spec.stream_float32 and L.model.use_graphs and L.model.head is L.model.embedding
    cache = L.model.new_cache(320)
    for ids in vm.prompts(L.cfg, (1, 2, 5, 70, 129, 300), seed=1):
        s = cache.open()
        close(L.model.step(cache, [s], [ids], want="all"), L.plain_logits(ids), dtype, f"{name} {len(ids)} tokens")
        cache.close(s)
    L.model.check_errors()
    cache.check()


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_residual_stream_after_every_layer(loaded, name):
    L = loaded(name, "float32")
    ids = vm.prompts(L.cfg, (50,), seed=2)[0]
    want, got = [], []
    plain.forward(L.cfg, L.w, ids, streams=want)
    blocks = L.model.blocks
    originals = [b.forward for b in blocks]
    try:
        for b, orig in zip(blocks, originals):
            b.forward = (lambda x, ctx, entry, orig=orig: (got.append(orig(x, ctx, entry)), got[-1])[1])
        cache = L.model.new_cache(64)
        L.model.step(cache, [cache.open()], [ids], want="last")
    finally:
        for b in blocks:
            del b.forward
    assert len(got) == len(want) == len(L.cfg["layers"])
    from pytorch_transformers_b200.parts.base import resolve
    for i, (a, b) in enumerate(zip(got, want)):
        a = resolve(K(), a)
        assert a.dtype == torch.float32 and row_errors(a, b).max() < 1e-5, f"layer {i}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_single_tokens(loaded, name, dtype):
    L = loaded(name, dtype)
    cache = L.model.new_cache(256)
    for n, head in ((100, 60), (34, 1), (200, 62)):        # the single tokens cross a page's border
        ids = vm.prompts(L.cfg, (n,), seed=n)[0]
        s = cache.open()
        rows = [L.model.step(cache, [s], [ids[:head]], want="all")]
        rows += [L.model.step(cache, [s], [[t]], want="last") for t in ids[head:]]
        close(torch.cat(rows), L.plain_logits(ids), dtype, f"{name} prompt of {head} then {n - head} single tokens")
        cache.close(s)
    L.model.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("portion", [2, 3, 17, 64])
def test_prompts_in_portions(loaded, name, dtype, portion):
    L = loaded(name, dtype)
    cache = L.model.new_cache(192)
    ids = vm.prompts(L.cfg, (150,), seed=portion)[0]
    s = cache.open()
    rows = [L.model.step(cache, [s], [ids[i:i + portion]], want="all") for i in range(0, len(ids), portion)]
    close(torch.cat(rows), L.plain_logits(ids), dtype, f"{name} in portions of {portion}")
    cache.close(s)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_a_long_prompt_in_two_portions(loaded, name, dtype):
    L = loaded(name, dtype)
    cache = L.model.new_cache(64 * 9)
    ids = vm.prompts(L.cfg, (530,), seed=12)[0]
    s = cache.open()
    got = torch.cat([L.model.step(cache, [s], [ids[:400]], want="all"), L.model.step(cache, [s], [ids[400:]], want="all")])
    close(got, L.plain_logits(ids), dtype, f"{name} 400 + 130 tokens")
    cache.close(s)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_batches_of_unequal_requests_on_a_small_cache(loaded, name, dtype):
    """Three batches one after the other on a cache that holds just one of them: slots and pages of one are
    used again by the next. Shorter requests end earlier."""
    L = loaded(name, dtype)
    cache = L.model.new_cache(64 * 7, max_slots=3)
    for seed, (lengths, heads) in enumerate([((130, 7, 66), (120, 2, 64)), ((3, 90, 65), (1, 64, 33)), ((75, 140, 80), (70, 129, 66))]):
        reqs = vm.prompts(L.cfg, lengths, seed=10 + seed)
        refs = [L.plain_logits(r) for r in reqs]
        slots = [cache.open() for _ in reqs]
        assert sorted(slots) == [0, 1, 2]
        out = L.model.step(cache, slots, [r[:h] for r, h in zip(reqs, heads)], want="last")
        live, t, got, want = [0, 1, 2], 0, [], []
        while True:
            for row, i in enumerate(live):
                got.append(out[row])
                want.append(refs[i][heads[i] + t - 1])
            for i in [i for i in live if heads[i] + t >= lengths[i]]:
                cache.close(slots[i])
            live = [i for i in live if heads[i] + t < lengths[i]]
            if not live:
                break
            out = L.model.step(cache, [slots[i] for i in live], [[reqs[i][heads[i] + t]] for i in live], want="last")
            t += 1
        close(torch.stack(got), torch.stack(want), dtype, f"{name} batch {seed}")
        cache.check()
        assert not cache.records
    L.model.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "ones", "wide"])
def test_long_decoding(loaded, name, dtype):
    L = loaded(name, dtype)
    cache = L.model.new_cache(64 * 12)
    reqs = vm.prompts(L.cfg, (330, 290), seed=5)
    refs = [L.plain_logits(r) for r in reqs]
    slots = [cache.open(), cache.open()]
    heads = (3, 1)
    out = [L.model.step(cache, slots, [r[:h] for r, h in zip(reqs, heads)], want="last")]
    L.model.record_steps(True)
    for t in range(289):
        out.append(L.model.step(cache, slots, [[reqs[0][3 + t]], [reqs[1][1 + t]]], want="last"))
    kinds = [r["kind"] for r in L.model.step_timings()]
    L.model.record_steps(False)
    assert kinds.count("graph") > 250            # the single-token steps were replayed graphs
    got = torch.stack(out)
    close(got[:, 0], refs[0][2:2 + 290], dtype, f"{name} long decoding, first")
    close(got[:, 1], refs[1][0:290], dtype, f"{name} long decoding, second")
    L.model.check_errors()
    cache.check()


def test_a_step_on_two_streams_and_on_one(loaded, monkeypatch):
    """Steps of few tokens may run the mixer beside the feed-forward on a second stream; whichever it is, the sums are
    float32 and the logits agree."""
    L = loaded("wide", "bfloat16")
    ids = vm.prompts(L.cfg, (90,), seed=21)[0]
    k = K()

    def run(two):
        monkeypatch.setattr(k, "decode_attention_fits_beside", lambda *a: two)
        cache = L.model.new_cache(128)
        s = cache.open()
        out = [L.model.step(cache, [s], [ids[:80]], want="last")]
        out += [L.model.step(cache, [s], [[t]], want="last") for t in ids[80:]]
        return torch.cat(out)

    a, b = run(True), run(False)
    close(a, L.plain_logits(ids)[79:], "bfloat16", "two streams")
    close(b, L.plain_logits(ids)[79:], "bfloat16", "one stream")
    assert row_errors(a, b).max() < 3e-3
    L.model.check_errors()


@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation_through_generate(loaded, name):
    L = loaded(name, "float32")
    prompts = vm.prompts(L.cfg, (9, 1, 30), seed=3)
    out = L.model.generate(prompts, max_new_tokens=12, do_sample=False, eos_token_id=None)
    for p, seq in zip(prompts, out):
        assert seq[:len(p)] == p and len(seq) == len(p) + 12
        ids = list(p)
        for tok in seq[len(p):]:
            logits = L.plain_logits(ids)[-1]
            top2 = logits.topk(2).values
            if float(top2[0] - top2[1]) > 1e-4:          # no test on a tie within float32 rounding
                assert int(logits.argmax()) == tok
            ids.append(tok)


def test_generation_with_sampling_and_stop_tokens_runs(loaded):
    L = loaded("mixed", "bfloat16")
    prompts = vm.prompts(L.cfg, (5, 40), seed=8)
    out = L.model.generate(prompts, max_new_tokens=20, do_sample=True, top_k=20, temperature=0.8, seed=1, eos_token_id=7)
    assert all(len(o) <= len(p) + 20 for o, p in zip(out, prompts))
    again = L.model.generate(prompts, max_new_tokens=20, do_sample=True, top_k=20, temperature=0.8, seed=1, eos_token_id=7)
    assert out == again


@pytest.mark.parametrize("dtype", DTYPES)
def test_random_model_from_config_and_from_folder_are_one_model(tmp_path, dtype):
    import pytorch_transformers_b200 as ptb
    cfg = ptb.VesidraConfig.from_dict(vm.CONFIGS["odd"])
    folder = ptb.write_random_model(cfg, seed=4, folder=str(tmp_path / "m"), dtype=tdtype(dtype))
    a = ptb.AutoModelForCausalLM.from_pretrained(folder, dtype=dtype)
    b = ptb.AutoModelForCausalLM.from_config(cfg, seed=4, dtype=dtype)
    ids = vm.prompts(vm.CONFIGS["odd"], (20,), seed=0)
    ca, cb = a.new_cache(64), b.new_cache(64)
    la, lb = a.step(ca, [ca.open()], ids, want="all"), b.step(cb, [cb.open()], ids, want="all")
    torch.testing.assert_close(la, lb, atol=0, rtol=0)
    assert torch.isfinite(la).all() and float(la.std()) > 0


def test_greedy_generation_from_the_command_line(tmp_path):
    """The library's command line on a Vesidra folder, as a child process: the design is found by the folder's
    configuration, and the tokens are the plain implementation's."""
    cfg = vm.CONFIGS["odd"]
    folder = vm.write_folder(tmp_path, "odd", seed=6)
    w = vm.torch_weights(cfg, 6)
    prompts = vm.prompts(cfg, (7, 20), seed=9)
    script = os.path.join(ROOT, "bin", "ptb200-cli")
    args = [sys.executable, script, "run-generation", "--model_name_or_path", folder, "--fp32", "--greedy", "--length", "8"]
    for q in prompts:
        args += ["--prompt_ids", ",".join(map(str, q))]
    done = subprocess.run(args, capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    recs = [json.loads(line) for line in done.stdout.splitlines() if line.startswith("{")]
    assert [r["prompt_ids"] for r in recs] == prompts
    for q, r in zip(prompts, recs):
        ids = list(q)
        assert len(r["generated_ids"]) == 8
        for tok in r["generated_ids"]:
            logits = plain.forward(cfg, w, ids)[-1]
            top2 = logits.topk(2).values
            if float(top2[0] - top2[1]) > 1e-4:          # no test on a tie within float32 rounding
                assert int(logits.argmax()) == tok
            ids.append(tok)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner_as_a_child_process(tmp_path, dtype):
    name = "mixed"
    cfg = vm.CONFIGS[name] if dtype == "float32" else vm.steady(vm.CONFIGS[name])
    folder = vm.write_folder(tmp_path, name, seed=2, bf16=(dtype == "bfloat16"), cfg=cfg)
    w = vm.torch_weights(cfg, 2)
    reqs = dict(zip("abc", vm.prompts(cfg, (70, 9, 40), seed=4)))
    refs = {kk: plain.forward(cfg, w, v) for kk, v in reqs.items()}
    heads = {"a": 64, "b": 6, "c": 40}
    steps = [{"step": 0, "entries": [{"id": i, "tokens": reqs[i][:heads[i]], "want": [0, heads[i] - 1]} for i in "abc"], "end": ["c"]}]
    expect = {0: [(i, p) for i in "abc" for p in (0, heads[i] - 1)]}
    for t in range(6):
        live = [i for i in "ab" if heads[i] + t < len(reqs[i])]
        steps.append({"step": t + 1, "entries": [{"id": i, "tokens": [reqs[i][heads[i] + t]], "want": [0]} for i in live],
                      "end": [i for i in live if heads[i] + t + 1 == len(reqs[i])]})
        expect[t + 1] = [(i, heads[i] + t) for i in live]
    out = str(tmp_path / "out")
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out,
                           "--max-tokens", "192"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True,
                          text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    got, want = [], []
    for step, rows in expect.items():
        arr = np.fromfile(os.path.join(out, f"{step}.f32"), dtype="<f4").reshape(-1, cfg["vocab"])
        assert arr.shape[0] == len(rows)
        got.append(torch.from_numpy(arr.copy()))
        want += [refs[i][p] for i, p in rows]
    close(torch.cat(got), torch.stack(want), dtype, "trace")
