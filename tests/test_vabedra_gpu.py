"""Vabedra on the GPU against the plain implementation (tests/plain_vabedra.py), in float32 and bfloat16.

First every mechanism alone: what enters the delta rule (short convolutions across portions, unit norms, decays, beta), the
recurrence as a kernel (walked and in chunks, a key far back that an open channel carries and a closed one has dropped, a
value that is written over, strong and weak decays), the delta rule as a part in both settings (whole, in portions, in
chunks, token by token, two sequences, a slot that is used again), the attention as a part (whole, in portions, single
tokens; one key that a query is aligned with, at a page's border, just inside and just outside the window and the kept first
tokens, in prompts and in single tokens; the cap; the added one of the softmax; the biases; the scaled frequencies), norms
after the sum in all their forms, the token input, the router and the clamped experts, a whole block. Then whole models of
several shapes: each request alone, the stream after every layer, a prompt and then single tokens, portions down to two
tokens, batches of unequal requests on a small cache whose slots and pages are used again, long decoding through replayed
graphs, greedy generation through ``generate`` and the command line, and the trace runner as a child process.
"""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_vabedra as plain
import vabedra_models as vm

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


class PartAlone:
    """A mixer or a block alone on a cache of its own, fed rows (and token ids) directly."""

    def __init__(self, spec, weights, dtype):
        from pytorch_transformers_b200.parts.base import BuildContext, make_part
        self.k, self.dt = K(), tdtype(dtype)
        self.part = make_part(BuildContext(torch.device("cuda"), self.dt, self.k), spec)
        for part in self.part.walk():
            decls = part.param_decls()
            if decls:
                part.bind({n: weights[part.spec.names[n]].to(device="cuda", dtype=torch.float32 if d.role == "vector" else self.dt)
                           for n, d in decls.items()})
        for part in self.part.walk():
            if hasattr(part, "after_bind"):
                part.after_bind()
        self.planners, self.table = [], None
        for part in self.part.walk():
            p = part.planner()
            for one in (p if isinstance(p, (list, tuple)) else [p]):
                if one is not None and one.plan_key not in [q.plan_key for q in self.planners]:
                    self.planners.append(one)

    def cache(self, max_tokens, max_slots=None):
        from pytorch_transformers_b200.cache.paged import Cache
        mixer = self.part.children.get("mixer", self.part)
        return Cache([(0, mixer.cache_need(), mixer.state_need())], max_tokens, self.dt, "cuda", max_slots=max_slots)

    def step(self, cache, slots, rows, ids=None):
        from pytorch_transformers_b200.engine.batch import StepContext
        from pytorch_transformers_b200.parts.base import ScheduleEntry, resolve
        ids = ids or [[0] * r.shape[0] for r in rows]
        ctx = StepContext(cache, slots, ids, 1 << 20, [[] for _ in rows], self.planners)
        ctx.begin_forward()
        ctx.token_table, ctx.status = self.table, torch.zeros(1, dtype=torch.int32, device="cuda")
        block = "mixer" in self.part.children
        x = torch.cat(rows).to(torch.float32 if block else self.dt).cuda().contiguous()
        y = resolve(self.k, self.part.forward(x, ctx, ScheduleEntry(0, 0)))
        ctx.commit()
        return list(y.double().cpu().split([r.shape[0] for r in rows]))

    def run_cut(self, cache, rows, cuts, ids=None):
        """One sequence fed in portions of the given sizes; returns all its output rows."""
        s, at, got = cache.open(), 0, []
        for n in cuts:
            got.append(self.step(cache, [s], [rows[at:at + n]], None if ids is None else [ids[at:at + n]])[0])
            at += n
        cache.close(s)
        return torch.cat(got)


def drawn(shapes, seed):
    rng = np.random.Generator(np.random.PCG64(seed))
    return {name: torch.from_numpy(vm.draw(name, shape, rng)) for name, shape in shapes.items()}


def config_of(layer, width, side=0, alpha=1.5):
    import pytorch_transformers_b200 as ptb
    raw = {"vocab": 50, "width": width, "norm": {"eps": 1e-5}, "postln_alpha": alpha, "layers": [layer]}
    if side:
        raw["token_side"] = {"dim": side}
    return ptb.VabedraConfig.from_dict(raw)


# ------------------------------------------------------------------------------------------------ the delta rule
def delta_part(m, width, channel, dtype, seed=0):
    from pytorch_transformers_b200.models.vabedra import _delta
    cfg = config_of({"type": "delta", "mixer": vm.delta(1, 1, 8, 8, 1), "mlp": None}, width)
    w = drawn(vm.delta_shapes(m, width, "m.", channel), seed)
    return PartAlone(_delta(cfg, m, "m.", channel), w, dtype), plain.sub(w, "m.")


DELTAS = [(vm.delta(4, 2, 24, 20, 4), False), (vm.delta(3, 3, 16, 40, 3, rank=8), True), (vm.delta(3, 1, 6, 10, 6, rank=5), True),
          (vm.delta(2, 1, 37, 11, 3), False), (vm.delta(1, 1, 8, 8, 1, rank=1), True), (vm.delta(4, 2, 64, 64, 4, rank=40), True),
          (vm.delta(4, 1, 64, 128, 4), False), (vm.delta(2, 2, 128, 64, 3, rank=16), True), (vm.delta(2, 1, 128, 128, 2), False),
          (vm.delta(1, 1, 200, 33, 2), False), (vm.delta(2, 2, 130, 16, 9, rank=3), True)]


def _did(v):
    m, channel = v
    return f"{m['heads']}h{m['kv_heads']}x{m['dim']}x{m['vdim']}{'c' if channel else ''}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,channel", DELTAS, ids=[_did(v) for v in DELTAS])
def test_what_enters_the_recurrence(m, channel, dtype):
    """Convolutions whose window reaches into earlier portions, silu, the norms' factors, the decays' logarithms, beta."""
    width, eps = 48, 1e-5
    mixer, w = delta_part(m, width, channel, dtype, seed=3)
    p, k, dt = mixer.part, K(), tdtype(dtype)
    g = torch.Generator().manual_seed(4)
    x = bf16_exact(torch.randn(40, width, generator=g))
    q, kk, v, beta = plain.delta_inputs(x, w, m)
    cache = mixer.cache(64, max_slots=2)
    cache.open()                                     # the sequence's slot is not the first
    s, at = cache.open(), 0
    from pytorch_transformers_b200.engine.batch import StepContext
    from pytorch_transformers_b200.parts.linear import linear
    entry = type("E", (), {"cache_entry": 0, "state_offset": 0})()
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    own = torch.tensor([h // (H // G) for h in range(H)])
    got = {n: [] for n in ("q", "k", "v", "l", "b")}
    for n in (1, 1, 2, 1, 3, 20, 1, 2, 9):
        ctx = StepContext(cache, [s], [[0] * n], 1, [[]], mixer.planners)
        proj = linear(k, x[at:at + n].to(dt).cuda().contiguous(), p.p_in)
        z = linear(k, proj[:, p.low_off:p.low_off + p.low], p.p_low, wide_out=True)[:, :H * d] if channel else None
        state = ctx.state_of(entry, p.state_need().numel)
        act, inv, logd, b = k.delta_prepare(proj, p.p_conv, state, ctx.dev["slots"], ctx.batch_c[0], p.p_a_log, p.p_dt_bias, H, G, d, vd,
                                            p.b_off, p.a_off, z, single_tokens=ctx.is_decode)
        ctx.commit()
        at += n
        act, inv = act.double().cpu(), inv.double().cpu()
        got["q"].append((act[:, :G * d].reshape(n, G, d) * inv[:, :G, None])[:, own])
        got["k"].append((act[:, G * d:2 * G * d].reshape(n, G, d) * inv[:, G:, None])[:, own])
        got["v"].append(act[:, 2 * G * d:].reshape(n, H, vd))
        got["l"].append(logd.double().cpu().reshape(n, H, -1).expand(n, H, d))
        got["b"].append(b.double().cpu())
    got = {n: torch.cat(v) for n, v in got.items()}
    unit = got["k"].norm(dim=-1)
    assert (unit - 1).abs().max() < 1e-3             # the root's 1e-6 is all that keeps a unit vector from length one
    for name, want in (("q", q), ("k", kk), ("v", v)):
        close(got[name].reshape(40, -1), want.reshape(40, -1), dtype, name, f32=5e-6, bf16=1.5e-2)
    close(got["b"], beta, dtype, "beta", f32=5e-6, bf16=1e-2)
    close(got["l"].exp().reshape(40, -1), plain.delta_decay(x, w, m).reshape(40, -1), dtype, "decays", f32=5e-6, bf16=1.5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,channel", [(vm.delta(4, 2, 24, 20, 4), False), (vm.delta(2, 2, 64, 40, 4, rank=5), True),
                                       (vm.delta(2, 1, 9, 6, 4, rank=3), True), (vm.delta(2, 1, 32, 32, 3), False),
                                       (vm.delta(1, 1, 144, 16, 4), False)], ids=lambda v: str(v) if isinstance(v, bool) else f"{v['dim']}x{v['conv']}")
def test_steps_of_many_tokens_form_the_same_inputs(m, channel, dtype):
    """Hundreds of tokens of several sequences in one step, after a first portion of a few tokens each: runs of tokens whose
    inputs reach into the portion before, that span two sequences and that end with the step."""
    width, lengths, heads = 48, [333, 9, 7, 420, 2], [3, 1, 2, 5, 1]
    mixer, w = delta_part(m, width, channel, dtype, seed=5)
    g = torch.Generator().manual_seed(6)
    xs = [bf16_exact(torch.randn(n, width, generator=g)).float() for n in lengths]
    cache = mixer.cache(64 * 20, max_slots=5)
    slots = [cache.open() for _ in xs]
    first = mixer.step(cache, slots, [x[:h] for x, h in zip(xs, heads)])
    second = mixer.step(cache, slots, [x[h:] for x, h in zip(xs, heads)])
    for x, a, b in zip(xs, first, second):
        close(torch.cat([a, b]), plain.delta_mixer(x.double(), w, m, 1e-5), dtype, f"{len(x)} tokens", f32=4e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,channel", DELTAS, ids=[_did(v) for v in DELTAS])
def test_delta_rule_whole_in_portions_in_chunks_and_token_by_token(m, channel, dtype):
    width = 48
    mixer, w = delta_part(m, width, channel, dtype, seed=m["dim"])
    g = torch.Generator().manual_seed(1)
    x = bf16_exact(torch.randn(330, width, generator=g)).float()
    ref = plain.delta_mixer(x.double(), w, m, 1e-5)
    cache = mixer.cache(64, max_slots=2)
    # 330 tokens at once run in chunks of 64 where the sizes allow (the last one short); 256 + 74 joins chunks and the walk
    for cuts in ([330], [256, 74], [100, 64, 2, 3, 17, 144], [1] * 40 + [290], [5] + [1] * 70 + [255]):
        close(mixer.run_cut(cache, x, cuts), ref, dtype, f"cuts {cuts[:6]}", f32=4e-5)
    # two sequences side by side, one ends early, and its slot is used again by a third
    y = bf16_exact(torch.randn(90, width, generator=g)).float()
    ref_y = plain.delta_mixer(y.double(), w, m, 1e-5)
    a, b = cache.open(), cache.open()
    out = mixer.step(cache, [a, b], [x[:70], y[:20]])
    got_x, got_y = [out[0]], [out[1]]
    for t in range(20, 25):
        out = mixer.step(cache, [a, b], [x[50 + t:51 + t], y[t:t + 1]])
        got_x.append(out[0]); got_y.append(out[1])
    cache.close(b)
    c = cache.open()
    assert c == b
    out = mixer.step(cache, [c, a], [y[:90], x[75:80]])
    close(torch.cat(got_x + [out[1]]), ref[:80], dtype, "first of two", f32=4e-5)
    close(torch.cat(got_y), ref_y[:25], dtype, "second of two", f32=4e-5)
    close(out[0], ref_y, dtype, "a slot that is used again starts from nothing", f32=4e-5)


class Rule:
    """The recurrence's kernel alone, on given queries, keys, values, logarithms of decays and betas."""

    def __init__(self, q, k, v, logd, beta, dtype, taps=3):
        self.n, self.G, self.d = q.shape
        self.H, self.vd, self.taps, self.dt = v.shape[1], v.shape[2], taps, tdtype(dtype)
        flat = lambda t: t.reshape(self.n, -1)
        self.act = torch.cat([flat(q), flat(k), flat(v)], 1).to(self.dt)
        self.logd, self.beta = logd.float(), beta.float()
        r = self.act.double()
        qr, kr = r[:, :self.G * self.d].reshape(self.n, self.G, -1), r[:, self.G * self.d:2 * self.G * self.d].reshape(self.n, self.G, -1)
        self.inv = torch.cat([1 / (qr.square().sum(-1) + 1e-6).sqrt(), 1 / (kr.square().sum(-1) + 1e-6).sqrt()], 1).float()
        own = torch.tensor([h // (self.H // self.G) for h in range(self.H)])
        i = self.inv.double()
        dec = self.logd.double().reshape(self.n, self.H, -1).exp().expand(self.n, self.H, self.d)
        self.inputs = ((qr * i[:, :self.G, None])[:, own], (kr * i[:, self.G:, None])[:, own],
                       r[:, 2 * self.G * self.d:].reshape(self.n, self.H, self.vd), dec, self.beta.double())

    def reference(self, lo=0, hi=None, state=None):
        return plain.delta_recurrence(*(t[lo:hi] for t in self.inputs), state)

    def need(self):
        return K().delta_state_floats(self.H, self.G, self.d, self.vd, self.taps)

    def cache(self, slots=4):
        from pytorch_transformers_b200.cache.paged import Cache
        from pytorch_transformers_b200.parts.base import StateNeed
        return Cache([(0, None, StateNeed(self.need()))], 64 * slots, self.dt, "cuda", max_slots=slots)

    def run(self, cache, slots, spans, chunked):
        """Rows spans[b] as the next tokens of slots[b]; (outputs [.., H * vd] per sequence)."""
        from pytorch_transformers_b200.engine.batch import StepContext
        from pytorch_transformers_b200.parts.recurrent import RecurrenceChunks

        class Always(RecurrenceChunks):     # chunks whatever the length
            def plan(self, ctx):
                from pytorch_transformers_b200.parts import recurrent
                was, recurrent.SCAN_CHUNKED_FROM = recurrent.SCAN_CHUNKED_FROM, 1
                try:
                    return super().plan(ctx)
                finally:
                    recurrent.SCAN_CHUNKED_FROM = was
        k = K()
        ctx = StepContext(cache, slots, [[0] * (b - a) for a, b in spans], 1, [[] for _ in spans], [Always()])
        plan, chunks = ctx.plan(RecurrenceChunks.plan_key), None
        if chunked:
            assert k.delta_chunks_take(self.act, self.d, self.vd)
            chunks = (plan.dev["chunk_seq"], plan.dev["chunk_q0"], plan.dev["seq_chunk0"], plan.facts["n_chunks"])
        pick = lambda t: torch.cat([t[a:b] for a, b in spans]).cuda().contiguous()
        entry = type("E", (), {"cache_entry": 0, "state_offset": 0})()
        state = ctx.state_of(entry, self.need())
        out = k.delta_rule(pick(self.act), pick(self.inv), pick(self.logd), pick(self.beta), state, ctx.dev["slots"], ctx.batch_c[0],
                           self.H, self.G, self.d, self.vd, self.taps, chunks)
        ctx.commit()
        return list(out.double().cpu().split([b - a for a, b in spans]))

    def left(self, cache, slot):
        off = (self.taps - 1) * (2 * self.G * self.d + self.H * self.vd)
        s = cache.state[slot, off:off + self.H * self.d * self.vd].double().cpu()
        return s.reshape(self.H, self.vd, self.d).transpose(1, 2)


def rule_case(H, G, d, vd, n, per_head, dtype, seed, strong=1.0):
    g = torch.Generator().manual_seed(seed)
    ld = -torch.rand(n, H if per_head else H * d, generator=g) * 0.2 * strong
    if not per_head:
        ld = ld.reshape(n, H, d)
        ld[:, :, 0], ld[:, :, 1] = 0.0, -9.0            # a channel that never fades, one that is gone after a token
        ld[:, H - 1, 2::3] *= 40.0
        ld = ld.reshape(n, H * d)
    return Rule(torch.randn(n, G, d, generator=g), torch.randn(n, G, d, generator=g), torch.randn(n, H, vd, generator=g), ld,
                torch.rand(n, H, generator=g), dtype)


@pytest.mark.parametrize("per_head", [False, True])
@pytest.mark.parametrize("H,G,d,vd", [(2, 1, 64, 64), (3, 3, 64, 128), (4, 2, 128, 64), (2, 2, 128, 128)])
@pytest.mark.parametrize("strong", [0.01, 1.0, 50.0])
def test_chunks_on_the_tensor_cores_against_the_walk_and_the_plain_rule(H, G, d, vd, per_head, strong):
    """Sequences of one token, of whole chunks and with a short last chunk, side by side, then a second portion from the
    state that the first left; far below bfloat16's rounding whatever the decays (float32 operands are split in two)."""
    rule = rule_case(H, G, d, vd, 700, per_head, "bfloat16", d + vd, strong)
    spans = [(0, 300), (300, 301), (301, 429), (429, 700)]
    for chunked, limit in ((True, 1e-4), (False, 2e-5)):
        cache = rule.cache()
        slots = [cache.open() for _ in spans]
        first = rule.run(cache, slots, spans, chunked)
        second = rule.run(cache, slots[::-1], [(100, 165), (0, 64), (5, 22), (600, 601)], chunked)
        for slot, (a, b), one, two, (c, e) in zip(slots, spans, first, second[::-1], [(600, 601), (5, 22), (0, 64), (100, 165)]):
            o, S = rule.reference(a, b)
            assert row_errors(one, o.reshape(b - a, -1)).max() < limit
            o2, S2 = rule.reference(c, e, S)
            assert row_errors(two, o2.reshape(e - c, -1)).max() < limit
            assert (rule.left(cache, slot) - S2).norm() < limit * S2.norm()


@pytest.mark.parametrize("dtype,chunked", [("float32", False), ("bfloat16", False), ("bfloat16", True)])
@pytest.mark.parametrize("n,back", [(700, 650), (300, 299), (130, 64), (65, 63), (17, 16), (16, 15), (40, 3), (2, 1), (1, 0)])
def test_a_far_key_on_an_open_channel_and_on_a_closed_one(n, back, dtype, chunked):
    """Two heads, one key at `back` tokens before the last query and none other near it: head 0 carries it on a channel that
    never fades and answers with its value whole; head 1's channel closes and the answer fades by exp(-0.05) a token."""
    d = vd = 64
    g = torch.Generator().manual_seed(n + back)
    q, k = torch.zeros(n, 2, d), torch.zeros(n, 2, d)
    q[:, :, 2:], k[:, :, 2:] = torch.randn(n, 2, d - 2, generator=g), torch.randn(n, 2, d - 2, generator=g)
    at = n - 1 - back
    k[at] = 0.0
    q[n - 1] = 0.0
    k[at, 0, 0] = k[at, 1, 1] = 3.0
    q[n - 1, 0, 0] = q[n - 1, 1, 1] = 3.0
    ld = torch.full((n, 2, d), -0.05)
    ld[:, 0, 0] = 0.0
    beta = torch.rand(n, 2, generator=g)
    beta[at] = 1.0
    rule = Rule(q, k, torch.randn(n, 2, vd, generator=g), ld.reshape(n, -1), beta, dtype)
    o, _ = rule.reference()
    for spans in ([(0, n)], [(0, n // 2), (n // 2, n)] if n > 1 else [(0, 1)]):
        cache = rule.cache()
        s = cache.open()
        got = torch.cat([rule.run(cache, [s], [sp], chunked)[0] for sp in spans])
        assert row_errors(got, o.reshape(n, -1)).max() < (1e-4 if chunked else 2e-5)
        last, v = got[n - 1].reshape(2, vd), rule.inputs[2][at]
        torch.testing.assert_close(last[0], v[0], atol=1e-4, rtol=1e-4)
        torch.testing.assert_close(last[1], v[1] * math.exp(-0.05 * back), atol=1e-4, rtol=1e-4)


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("first,second", [(0, 1), (3, 15), (3, 16), (14, 40), (5, 63), (5, 64), (60, 130)])
def test_a_value_is_written_over_at_the_same_key(first, second, chunked):
    """The same key twice with beta 1 and no decay: after the second write the first value is gone. Both writes lie in one
    sub-block, in two, in two chunks."""
    n, d, vd = 200, 128, 64
    g = torch.Generator().manual_seed(first + second)
    q, k = torch.zeros(n, 1, d), torch.zeros(n, 1, d)
    k[:, 0, 1:] = torch.randn(n, d - 1, generator=g)
    k[first], k[second] = 0.0, 0.0
    k[first, 0, 0] = k[second, 0, 0] = 2.0
    q[:, 0, 0] = 1.0
    beta = torch.full((n, 1), 0.5)
    beta[first] = beta[second] = 1.0
    rule = Rule(q, k, torch.randn(n, 1, vd, generator=g), torch.zeros(n, d), beta, "bfloat16")
    cache = rule.cache()
    got = rule.run(cache, [cache.open()], [(0, n)], chunked)[0]
    v = rule.inputs[2][:, 0]
    for t in (0, first, second - 1, second, second + 1, n - 1):
        want = torch.zeros(vd, dtype=F64) if t < first else (v[first] if t < second else v[second])
        torch.testing.assert_close(got[t], want, atol=2e-4, rtol=2e-4)


# ------------------------------------------------------------------------------------------------ the attention
def attention_part(m, width, dtype, w):
    from pytorch_transformers_b200.models.vabedra import _attention
    cfg = config_of({"type": "delta", "mixer": vm.delta(1, 1, 8, 8, 1), "mlp": None}, width)
    return PartAlone(_attention(cfg, m, "m."), w, dtype)


ATTENTIONS = [vm.att(6, 2, 24, 20, 0.6, softcap=4.0, window=33, keep=5, rot=(8, 10000.0, 4.0, 1.0, 3.0, 64)),
              vm.att(5, 5, 10, 14, 0.4, window=129, keep=70, rot=(6, 10000.0, 2.0, 0.5, 8.0, 200)),
              vm.att(8, 2, 64, 64, 0.2, softcap=15.0, window=130, keep=4, rot=(32, 100000.0, 8.0, 1.0, 4.0, 100)),
              vm.att(2, 1, 128, 128, 0.1, softcap=30.0, rot=(128, 500.0)),
              vm.att(1, 1, 16, 16, 1.0 / 16, softcap=1.0, window=1, keep=1, rot=(2, 10.0)),
              vm.att(2, 2, 96, 32, 0.15, softcap=9.0, window=70, keep=0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", ATTENTIONS, ids=lambda m: f"{m['heads']}h{m['kv_heads']}x{m['dim']}x{m['vdim']}")
def test_attention_whole_in_portions_and_single_tokens(m, dtype):
    width = 40
    w = drawn(vm.attention_shapes(m, width, "m."), m["dim"])
    mixer = attention_part(m, width, dtype, w)
    g = torch.Generator().manual_seed(3)
    x = bf16_exact(torch.randn(300, width, generator=g)).float()
    ref = plain.attention_mixer(x.double(), plain.sub(w, "m."), m, 1e-5)
    no_bias = plain.attention_mixer(x.double(), {k: v * (0 if k.endswith(".b") else 1) for k, v in plain.sub(w, "m.").items()}, m, 1e-5)
    assert row_errors(no_bias, ref).median() > 0.1           # the biases show
    cache = mixer.cache(384)
    for cuts in ([300], [130, 170], [64, 2, 3, 17, 214], [120] + [1] * 100 + [80], [1] * 80 + [220]):
        close(mixer.run_cut(cache, x, cuts), ref, dtype, f"cuts {cuts[:6]}", f32=2e-5)
        cache.check()
    y = bf16_exact(torch.randn(150, width, generator=g)).float()
    ref_y = plain.attention_mixer(y.double(), plain.sub(w, "m."), m, 1e-5)
    a, b = cache.open(), cache.open()
    out = mixer.step(cache, [a, b], [x[:100], y[:62]])
    got_x, got_y = [out[0]], [out[1]]
    for t in range(80):
        out = mixer.step(cache, [a, b], [x[100 + t:101 + t], y[62 + t:63 + t]])
        got_x.append(out[0]); got_y.append(out[1])
    close(torch.cat(got_x), ref[:180], dtype, "first of two", f32=2e-5)
    close(torch.cat(got_y), ref_y[:142], dtype, "second of two", f32=2e-5)


def copying_weights(m):
    """Weights under which the mixer's input row is (q of every head | k of every K/V head | v): the test writes queries,
    keys and values directly. No biases, gains of one, the output projection is the identity."""
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    width = (H + G) * d + G * vd
    eye = torch.eye(width)
    return {"m.q": eye[:H * d], "m.k": eye[H * d:(H + G) * d], "m.v": eye[(H + G) * d:], "m.o": torch.eye(H * vd), "m.q.b": torch.zeros(H * d),
            "m.k.b": torch.zeros(G * d), "m.v.b": torch.zeros(G * vd), "m.q.norm": torch.ones(d), "m.k.norm": torch.ones(d)}, width


def needle_rows(m, n, at, g):
    """Random queries, keys and values; the last query and the key at `at` lie along one direction (in the entries that are
    not rotated), so that their score stands out."""
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    x = torch.randn(n, (H + G) * d + G * vd, generator=g)
    lo = (m.get("rot") or {}).get("dims", 0)
    direction = torch.zeros(d)
    direction[lo:] = torch.randn(d - lo, generator=g)
    x[n - 1, :H * d] = direction.repeat(H)
    x[at, H * d:(H + G) * d] = direction.repeat(G)
    return bf16_exact(x).float()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,window,keep,dims", [(24, 33, 5, 8), (64, 130, 4, 32), (64, 64, 64, 0), (128, 70, 0, 64), (72, 129, 70, 24)])
def test_attention_sees_a_key_just_inside_and_not_just_outside(d, window, keep, dims, dtype):
    """One aligned key at the window's last place, one further, at the last kept position and the one after it, at a page's
    border and at position 0; the query is the last token of a prompt, of a second portion, or a single token. The cap of 12
    lies above the needle's score and below what the scale alone would give."""
    m = vm.att(2, 1, d, d, 2.0 / math.sqrt(d), softcap=12.0, window=window, keep=keep, rot=(dims, 10000.0, 2.0, 1.0, 4.0, 90) if dims else None)
    w, width = copying_weights(m)
    mixer = attention_part(m, width, dtype, w)
    n = window + keep + 150
    cache = mixer.cache(64 * ((n + 63) // 64 + 1))
    places = {n - window: True, n - window - 1: keep > n - window - 1, 0: keep > 0, n - 1: True, n - 2: window > 1,
              64: keep > 64 or n - 1 - 64 < window, 63: keep > 63 or n - 1 - 63 < window}
    if keep:
        places.update({keep - 1: True, keep: n - 1 - keep < window})
    for at, seen in places.items():
        x = needle_rows(m, n, at, torch.Generator().manual_seed(at + d))
        ref = plain.attention_mixer(x.double(), plain.sub(w, "m."), m, 1e-5)
        value = x[at, -d:].double()
        for cuts in ([n], [n - 70, 70], [n - 30] + [1] * 30):
            got = mixer.run_cut(cache, x, cuts)
            close(got, ref, dtype, f"key at {at}, cuts {cuts[:2]}", f32=2e-5)
            cache.check()
            hit = (got[-1, :d] - value).norm() < 0.5 * value.norm()
            if d >= 64:
                assert hit == seen, f"key at {at} of {n}, window {window}, keep {keep}: seen {hit}, expected {seen}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,at", [(700, 3), (300, 63), (300, 64), (130, 127), (129, 128), (65, 64), (2, 0)])
def test_attention_without_a_window_finds_one_key_far_back(n, at, dtype):
    m = vm.att(2, 2, 64, 64, 0.5, softcap=25.0)
    w, width = copying_weights(m)
    mixer = attention_part(m, width, dtype, w)
    x = needle_rows(m, n, at, torch.Generator().manual_seed(n))
    ref = plain.attention_mixer(x.double(), plain.sub(w, "m."), m, 1e-5)
    cache = mixer.cache(768)
    for cuts in ([n], [n - 1, 1], [max(1, n - 40)] + [1] * min(40, n - 1)):
        got = mixer.run_cut(cache, x, cuts)
        close(got, ref, dtype, f"cuts {cuts[:3]}", f32=2e-5)
        value = x[at, -128:].double()
        assert (got[-1] - value).norm() < 0.1 * value.norm()


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_added_one_takes_weight_when_every_score_is_low(dtype):
    """Scores far below 0: the added one holds nearly all the weight and the output shrinks to nearly nothing; scores far
    above 0: it holds nearly none; and a cap binds both."""
    for cap, low_left in ((None, 1e-4), (2.0, 1.0)):
        m = vm.att(1, 1, 16, 16, 1.0, softcap=cap, window=1000)
        w, width = copying_weights(m)
        mixer = attention_part(m, width, dtype, w)
        g = torch.Generator().manual_seed(0)
        x = torch.randn(40, width, generator=g)
        direction = torch.randn(16, generator=g)
        x[:, :16], x[:, 16:32] = direction, -direction           # every score = -16
        x = bf16_exact(x).float()
        cache = mixer.cache(64)
        low = mixer.run_cut(cache, x, [40])
        want = plain.attention_mixer(x.double(), plain.sub(w, "m."), m, 1e-5)
        close(low, want, dtype, "low scores")
        assert float(low[0].abs().max()) < low_left
        share = math.exp(-16) if cap is None else 1 / (1 + math.exp(2 * math.tanh(8)))       # one key: e^s / (1 + e^s)
        torch.testing.assert_close(low[0], x[0, 32:].double() * share, atol=1e-2 * share, rtol=2e-2)
        x[:, 16:32] = x[:, :16]                                  # every score = +16
        close(mixer.run_cut(cache, x, [40]), plain.attention_mixer(x.double(), plain.sub(w, "m."), m, 1e-5), dtype, "high scores")


def test_scaled_frequencies_reach_the_table():
    """Kept, mixed and divided frequencies of one table, and the angles at far positions."""
    from pytorch_transformers_b200.parts.base import BuildContext, PartSpec, make_part
    rot = {"dims": 40, "base": 700.0, "scaling": {"factor": 6.0, "low": 1.5, "high": 5.0, "original": 130}}
    part = make_part(BuildContext(torch.device("cuda"), torch.float32, K()),
                     PartSpec("position", "rotary", {"head_dim": 48, "theta": 700.0, "rotary_dim": 40, "bands": rot["scaling"]}))
    want = torch.tensor(plain.frequencies(rot), dtype=F64)
    base = torch.tensor(plain.frequencies(dict(rot, scaling=None)), dtype=F64)
    ratio = want / base
    assert (ratio == 1).any() and (ratio - 1 / 6.0).abs().min() < 1e-12 and ((ratio < 0.99) & (ratio > 0.18)).any()
    torch.testing.assert_close(part.rotation().double().cpu(), want, atol=0, rtol=1e-7)
    pos = torch.tensor([0, 1, 130, 5000], dtype=torch.int32).cuda()
    cos, sin = K().rope_table(pos, part.rotation())
    a = pos.double().cpu()[:, None] * part.rotation().double().cpu()
    torch.testing.assert_close(cos.double().cpu(), torch.cos(a), atol=5e-4, rtol=0)
    torch.testing.assert_close(sin.double().cpu(), torch.sin(a), atol=5e-4, rtol=0)


# ------------------------------------------------------------------------------------------------ norms after the sum
@pytest.mark.parametrize("copy_dtype", DTYPES)
@pytest.mark.parametrize("width", [192, 53, 2050, 1])
def test_norms_after_the_sum(width, copy_dtype):
    k, cd = K(), tdtype(copy_dtype)
    g = torch.Generator().manual_seed(width)
    rn = lambda *s: torch.randn(*s, generator=g)
    n = 9
    x, a, b = rn(n, width) * 3, rn(n, width), rn(n, width) * 0.01
    gain, ga, gb = 1 + 0.3 * rn(width), 1 + 0.3 * rn(width), rn(width)
    D = lambda t: t.double()
    rms = lambda t, eps: plain.rms(D(t), eps)

    def check(got, want, what):
        stream, copy = got
        assert stream.dtype == torch.float32 and copy.dtype == cd
        close(stream, want, "float32", what, f32=2e-6)
        torch.testing.assert_close(copy, stream.to(cd), atol=0, rtol=0)
    c = lambda t: t.cuda()
    check(k.post_norm(c(x), c(a), c(gain), 1.7, 1e-3, cd), rms(1.7 * D(x) + D(a), 1e-3) * D(gain), "a branch")
    a16 = a.bfloat16()
    check(k.post_norm(c(x), c(a16), c(gain), 0.5, 1e-5, cd), rms(0.5 * D(x) + D(a16), 1e-5) * D(gain), "a bfloat16 branch")
    want = rms(2.5 * D(x) + 0.5 * (rms(a, 1e-4) * D(ga) + rms(b, 1e-4) * D(gb)), 1e-5) * D(gain)
    check(k.post_norm_pair(c(x), c(a), c(b), c(ga), c(gb), 0.5, 1e-4, c(gain), 2.5, 1e-5, cd), want, "a pair")
    top = 3
    rows, weights = rn(n * top, width), torch.rand(n, top, generator=g)
    perm = torch.randperm(n * top, generator=g).int()
    y = (D(weights)[:, :, None] * D(rows)[perm.long()].reshape(n, top, width)).sum(1)
    check(k.post_norm_experts(c(x), c(rows), c(perm), c(weights), c(gain), 1.3, 1e-5, cd), rms(1.3 * D(x) + y, 1e-5) * D(gain), "experts")
    check(k.norm_add(c(x), c(a), c(gain), 1e-2, cd), D(x) + rms(a, 1e-2) * D(gain), "the sum of a normed branch")
    torch.testing.assert_close(k.round_rows(c(x), cd), c(x).to(cd), atol=0, rtol=0)


def test_token_gate_reads_the_tokens_own_columns():
    k = K()
    g = torch.Generator().manual_seed(1)
    for dtype in DTYPES:
        table = torch.randn(30, 21, generator=g).to(tdtype(dtype))
        z, ids = torch.randn(11, 7, generator=g) * 2, torch.randint(0, 30, (11,), generator=g).int()
        for first in (0, 7, 14):
            out = k.token_gate(z.cuda(), ids.cuda(), table.cuda(), first, 7, 32)
            want = plain.gelu_tanh(z.double()) * table.double()[ids.long(), first:first + 7]
            close(out[:, :7], want, dtype, f"columns from {first}", f32=2e-6, bf16=4e-3)
            assert float(out[:, 7:].abs().max()) == 0.0
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        k.token_gate(z.cuda(), torch.full((11,), 30, dtype=torch.int32).cuda(), table.cuda(), 0, 7, 32, status)
        assert int(status) == 1


# ------------------------------------------------------------------------------------------------ the feed-forward
@pytest.mark.parametrize("n,top", [(16, 3), (5, 2), (1, 1), (64, 6), (7, 7)])
def test_router_scores_without_and_chooses_with_the_correction(n, top):
    k = K()
    g = torch.Generator().manual_seed(n)
    for tokens in (1, 7, 700):
        h, wr = torch.randn(tokens, 24, generator=g), torch.randn(n, 24, generator=g) * 0.5
        corr = torch.randn(n, generator=g) * 0.3
        ids, weights = plain.route(h.double(), wr.double(), corr.double(), top)
        got_ids, got_w = k.route(h.cuda(), wr.cuda(), corr.cuda(), 1, 1, top, 1.0, "softmax")
        # a choice may differ where two scores are within float32 rounding of each other
        same = (got_ids.cpu().long().sort(1).values == ids.sort(1).values).all(1)
        assert same.double().mean() > 0.99
        rows = same.nonzero().flatten()
        order = got_ids.cpu().long()[rows].argsort(1)
        torch.testing.assert_close(got_w.double().cpu()[rows].gather(1, order), weights[rows].gather(1, ids[rows].argsort(1)), atol=1e-6, rtol=1e-5)
        if tokens == 700 and n == 16:
            assert not torch.equal(ids.sort(1).values, plain.route(h.double(), wr.double(), 0 * corr.double(), top)[0].sort(1).values)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp,width", [(vm.moe(6, 2, 40, 0.7), 96), (vm.moe(5, 2, 18, 0.9), 52), (vm.moe(1, 1, 16, 1.0), 32),
                                       (vm.moe(16, 4, 64, 2.0), 128), (vm.moe(9, 9, 24, 0.3), 64)])
def test_clamped_experts(mlp, width, dtype):
    from pytorch_transformers_b200.models.vabedra import _feed_forward
    from pytorch_transformers_b200.parts.base import BuildContext, make_part
    layer = {"type": "delta", "mixer": vm.delta(1, 1, 8, 8, 1), "mlp": mlp}
    cfg = {"vocab": 8, "width": width, "layers": [layer]}
    w = {n: torch.from_numpy(v) for n, v in vm.make_weights(cfg, width).items()}
    dt = tdtype(dtype)
    part = make_part(BuildContext(torch.device("cuda"), dt, K()), _feed_forward(config_of(layer, width), 0))
    part.bind({n: w[part.spec.names[n]].to(device="cuda", dtype=torch.float32 if d.role == "vector" else dt)
               for n, d in part.param_decls().items()})
    g = torch.Generator().manual_seed(5)
    for tokens in (1, 9, 300):
        h = bf16_exact(1.5 * torch.randn(tokens, width, generator=g)).float()
        want = plain.moe(h.double(), plain.sub(w, "l0.mlp."), mlp)
        unclamped = plain.moe(h.double(), plain.sub(w, "l0.mlp."), dict(mlp, expert=dict(mlp["expert"], limit=1e9)))
        assert row_errors(unclamped, want).median() > 0.02          # the clamps bind
        close(part.forward(h.to(dt).cuda(), None), want, dtype, f"{tokens} tokens", f32=2e-5)
        rows, where, weights = part.forward_rows(h.to(dt).cuda(), None)
        summed = (weights[:, :, None] * rows[where.long()].reshape(tokens, -1, width)).sum(1)
        close(summed, want, dtype, "rows", f32=2e-5)


# ------------------------------------------------------------------------------------------------ a block
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,i", [("mixed", 0), ("mixed", 1), ("mixed", 2), ("odd", 0), ("ones", 0), ("wide", 0), ("wide", 2)])
def test_a_block_alone(name, i, dtype):
    """Mixer, norms after the sums, experts and token input together, in one step and in portions."""
    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200.models.vabedra import vabedra_block
    raw = vm.CONFIGS[name] if dtype == "float32" else vm.steady(vm.CONFIGS[name])
    w = {n: torch.from_numpy(v) for n, v in vm.make_weights(raw, 7).items()}
    block = PartAlone(vabedra_block(ptb.VabedraConfig.from_dict(raw), i), w, dtype)
    side = (raw.get("token_side") or {}).get("dim", 0)
    if side:
        block.table = w["side.embed"].to(device="cuda", dtype=tdtype(dtype))
    g = torch.Generator().manual_seed(8)
    x = bf16_exact(torch.randn(280, raw["width"], generator=g)).float()
    ids = torch.randint(0, raw["vocab"], (280,), generator=g).tolist()
    layer, eps, alpha, p = raw["layers"][i], raw["norm"]["eps"], raw["postln_alpha"], f"l{i}."
    mix = plain.delta_mixer if layer["type"] == "delta" else plain.parallel_mixer
    want = plain.rms(alpha * x.double() + mix(x.double(), plain.sub(w, p + "mix."), layer["mixer"], eps), eps) * w[p + "norm1"].double()
    if layer["mlp"] is not None:
        want = plain.rms(alpha * want + plain.moe(want, plain.sub(w, p + "mlp."), layer["mlp"]), eps) * w[p + "norm2"].double()
    if side:
        want = plain.token_side(want, w["side.embed"].double()[torch.tensor(ids), i * side:(i + 1) * side], plain.sub(w, p + "side."), eps)
    cache = block.cache(320)
    for cuts in ([280], [66, 2, 1, 1, 210], [100] + [1] * 30 + [150]):
        close(block.run_cut(cache, x, cuts, ids), want, dtype, f"{name} layer {i}, cuts {cuts[:4]}", f32=5e-5)


# ------------------------------------------------------------------------------------------------ whole models
class Loaded:
    def __init__(self, tmp, name, dtype):
        import pytorch_transformers_b200 as ptb
        # bfloat16 models run routers that choose every expert (vabedra_models.steady says why)
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
    assert L.model.spec.stream_float32 and L.model.use_graphs
    cache = L.model.new_cache(320)
    for ids in vm.prompts(L.cfg, (1, 2, 5, 70, 129, 300), seed=1):
        s = cache.open()
        close(L.model.step(cache, [s], [ids], want="all"), L.plain_logits(ids), dtype, f"{name} {len(ids)} tokens")
        cache.close(s)
    L.model.check_errors()
    cache.check()


def test_residual_stream_after_every_layer(loaded):
    L = loaded("mixed", "float32")
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
    assert len(got) == len(want) == 4
    from pytorch_transformers_b200.parts.base import resolve
    for i, (a, b) in enumerate(zip(got, want)):
        a = resolve(K(), a)
        assert a.dtype == torch.float32 and row_errors(a, b).max() < 1e-5, f"layer {i}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_single_tokens(loaded, name, dtype):
    L = loaded(name, dtype)
    cache = L.model.new_cache(256)
    for n, head in ((100, 60), (34, 1), (200, 62)):        # the single tokens cross a page's border and pass the windows
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
    """Two batches one after the other on a cache that holds just one of them: slots and pages of the first are
    used again by the second, whose sequences must start from empty state. Shorter requests end earlier."""
    L = loaded(name, dtype)
    cache = L.model.new_cache(64 * 5, max_slots=3)
    for seed, (lengths, heads) in enumerate([((130, 7, 66), (120, 2, 64)), ((3, 90, 65), (1, 64, 33))]):
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
    cfg = ptb.VabedraConfig.from_dict(vm.CONFIGS["odd"])
    folder = ptb.write_random_model(cfg, seed=4, folder=str(tmp_path / "m"), dtype=tdtype(dtype))
    a = ptb.AutoModelForCausalLM.from_pretrained(folder, dtype=dtype)
    b = ptb.AutoModelForCausalLM.from_config(cfg, seed=4, dtype=dtype)
    ids = vm.prompts(vm.CONFIGS["odd"], (20,), seed=0)
    ca, cb = a.new_cache(64), b.new_cache(64)
    la, lb = a.step(ca, [ca.open()], ids, want="all"), b.step(cb, [cb.open()], ids, want="all")
    torch.testing.assert_close(la, lb, atol=0, rtol=0)
    assert torch.isfinite(la).all() and float(la.std()) > 0


def test_greedy_generation_from_the_command_line(tmp_path):
    """The library's command line on a Vabedra folder, as a child process: the design is found by the folder's
    configuration, and the tokens are the plain implementation's."""
    cfg = vm.CONFIGS["odd"]
    folder = vm.write_folder(tmp_path, "odd", seed=6)
    w = vm.torch_weights(cfg, 6)
    prompts = vm.prompts(cfg, (7, 20), seed=9)
    script = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "ptb200-cli")
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
