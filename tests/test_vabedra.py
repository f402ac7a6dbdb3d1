"""Vabedra without a GPU: configuration and registry, the spec (tensor names and shapes, pages for the attention beside state
for the delta rule in one cache entry, the shared table of token inputs), refused configurations and parts, and the plain
implementation's own consistency (the rule carried from one half of a sequence to the next and as a solve of linear equations,
a value written over, the convolution's window, the scaled frequencies' three bands, the added one of the softmax)."""
import json
import math

import pytest
import torch

import plain_vabedra as plain
import vabedra_models as vm

F64 = torch.float64


def test_registry_finds_the_design_by_its_architecture_string(tmp_path):
    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200.config.registry import lookup
    folder = vm.write_folder(tmp_path, "mixed")
    cfg = ptb.AutoConfig.from_pretrained(folder)
    assert isinstance(cfg, ptb.VabedraConfig) and cfg.vocab == 211 and cfg.width == 96 and len(cfg.layers) == 4
    assert cfg.vocab_size == 211 and cfg.hidden_size == 96 and cfg.num_hidden_layers == 4
    assert lookup({"architecture": "Vabedra"}).model_type == "vabedra"
    back = ptb.VabedraConfig.from_dict(json.loads(json.dumps(cfg.to_dict())))
    assert back.layers == cfg.layers and back.token_side == cfg.token_side and back.postln_alpha == cfg.postln_alpha


@pytest.mark.parametrize("name", sorted(vm.CONFIGS))
def test_spec_names_every_tensor_and_states_every_need(name):
    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200.models.vabedra import vabedra_spec
    raw = vm.CONFIGS[name]
    cfg = ptb.VabedraConfig.from_dict(raw)
    spec = vabedra_spec(cfg)
    assert spec.stream_float32 and spec.head_name == "head" and spec.embedding_scale == raw["embedding"]["scale"]
    model = ptb.CausalLM(spec, cfg, device="cpu", dtype=torch.float32)
    table, want = model.param_table(), vm.tensor_shapes(raw)
    assert set(table) == set(want)
    for tensor, (_, _, decl) in table.items():
        assert tuple(decl.shape) == tuple(want[tensor]), tensor
    for (entry, c, s), layer in zip(model.cache_needs(), raw["layers"]):
        m = layer["mixer"]
        r = m if layer["type"] == "delta" else m["right"]
        channels = 2 * r["kv_heads"] * r["dim"] + r["heads"] * r["vdim"]
        exact = (r["conv"] - 1) * channels + r["heads"] * r["dim"] * r["vdim"]
        assert s.numel % 4 == 0 and exact <= s.numel < exact + 4
        if layer["type"] == "delta":
            assert c is None
        else:
            mask, l = m["left"].get("mask") or {}, m["left"]
            assert (c.kind, c.window, c.keep_first, c.kv_heads, c.head_dim, c.v_head_dim) == \
                ("window" if mask.get("size") else "full", mask.get("size", 0), mask.get("keep_first", 0), l["kv_heads"], l["dim"], l["vdim"])
    assert model.use_graphs


def test_low_ranks_may_come_from_the_checkpoint_alone():
    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200.models.vabedra import vabedra_spec
    from pytorch_transformers_b200.weights.random_init import random_tensor
    raw = json.loads(json.dumps(vm.CONFIGS["odd"]))
    del raw["layers"][0]["mixer"]["right"]["rank"]
    cfg = ptb.VabedraConfig.from_dict(raw)
    table = ptb.CausalLM(vabedra_spec(cfg), cfg, device="cpu", dtype=torch.float32).param_table()
    assert tuple(table["l0.mix.right.a1"][2].shape) == (-1, 52) and tuple(table["l0.mix.right.g2"][2].shape) == (30, -1)
    with pytest.raises(ValueError):
        random_tensor("l0.mix.right.a1", table["l0.mix.right.a1"][2], 0, "cpu", torch.float32)


def test_projections_are_put_together_at_whole_words():
    """The delta rule's one input matrix: q, k, v, gate, beta, decay, then the low-rank matrices at a multiple of 8 columns,
    padded to 32; the second matrices block by block. Two ranks that differ are taken."""
    from pytorch_transformers_b200 import kernels
    from pytorch_transformers_b200.parts.base import BuildContext, PartSpec, make_part
    build = BuildContext(torch.device("cpu"), torch.float32, kernels)
    p = {"hidden": 5, "heads": 3, "kv_heads": 1, "dim": 2, "vdim": 3, "taps": 2}
    part = make_part(build, PartSpec("mixer", "delta_rule", dict(p, decay="channel", gate="low_rank", gate_act="sigmoid")))
    g = torch.Generator().manual_seed(0)
    t = {n: torch.randn(*s, generator=g) for n, s in {"q": (2, 5), "k": (2, 5), "v": (9, 5), "q_conv": (2, 2), "k_conv": (2, 2),
         "v_conv": (9, 2), "b": (3, 5), "a_log": (3,), "norm": (3,), "o": (5, 9), "a1": (4, 5), "a2": (6, 4), "dt_bias": (6,),
         "g1": (7, 5), "g2": (9, 7)}.items()}
    part.bind(dict(t))
    assert part.low_off == 16 and part.low == 32 and part.in_rows() == 48 and part.in_weight().shape == (48, 5)
    x = torch.randn(4, 5, generator=g)
    proj = x @ part.in_weight().T
    low = proj[:, part.low_off:] @ part.p_low.T
    torch.testing.assert_close(low[:, :6], (x @ t["a1"].T) @ t["a2"].T)
    torch.testing.assert_close(low[:, 6:], (x @ t["g1"].T) @ t["g2"].T)
    torch.testing.assert_close(proj[:, part.b_off:part.b_off + 3], x @ t["b"].T)
    head = make_part(build, PartSpec("mixer", "delta_rule", dict(p)))
    t.update(a=torch.randn(3, 5, generator=g), g=torch.randn(9, 5, generator=g), dt_bias=torch.randn(3, generator=g))
    head.bind({n: t[n] for n in head.param_decls()})
    proj = x @ head.in_weight().T
    assert proj.shape[1] % 8 == 0
    torch.testing.assert_close(proj[:, head.a_off:head.a_off + 3], x @ t["a"].T)
    torch.testing.assert_close(proj[:, head.g_off:head.g_off + 9], x @ t["g"].T)
    with pytest.raises(ValueError):
        part.bind(dict(t, a2=torch.zeros(6, 5)))


def _with(name, **changes):
    cfg = json.loads(json.dumps(vm.CONFIGS[name]))
    for path, value in changes.items():
        at, keys = cfg, path.split("__")
        for k in keys[:-1]:
            at = at[int(k)] if k.isdigit() else at[k]
        at[keys[-1]] = value
    return cfg


@pytest.mark.parametrize("bad", [
    dict(vocab=0), dict(width=-1), dict(layers=[]), dict(norm={"eps": 0}), dict(layers__0__type="conv"), dict(token_side={"dim": 0}),
    dict(embedding={"scale": "x"}), dict(layers__0__mixer__heads=0), dict(layers__0__mixer__kv_heads=3), dict(layers__0__mixer__conv=0),
    dict(layers__1__mixer__left__scale=0), dict(layers__1__mixer__left__softcap=-1.0), dict(layers__1__mixer__left__kv_heads=4),
    dict(layers__1__mixer__left__rot__dims=7), dict(layers__1__mixer__left__rot__dims=26),
    dict(layers__1__mixer__left__rot__scaling={"factor": 2.0}), dict(layers__1__mixer__left__mask__size=-1),
    dict(layers__1__mixer__right={}), dict(layers__1__mixer__left=None), dict(layers__0__mlp__router__top=7),
    dict(layers__0__mlp__expert={"ff": 8}), dict(layers__0__mlp__expert={"ff": 8, "limit": -1.0}), dict(layers__0__mlp__kind="dense"),
])
def test_configurations_that_cannot_be_built_are_refused(bad):
    import pytorch_transformers_b200 as ptb
    with pytest.raises(ptb.ConfigError):
        ptb.VabedraConfig.from_dict(_with("mixed", **bad))


def test_keys_that_the_design_does_not_know_and_whole_numbers_written_as_floats_are_taken():
    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200.models.vabedra import vabedra_spec
    noted = _with("mixed", seed=11, layers__0__note="first", layers__1__mixer__left__mask={"size": 33.0, "keep_first": 5.0},
                  layers__1__mixer__left__rot__dims=8.0)
    a, b = vabedra_spec(ptb.VabedraConfig.from_dict(noted)), vabedra_spec(ptb.VabedraConfig.from_dict(_with("mixed")))
    assert [blk.children["mixer"].params for blk in a.blocks] == [blk.children["mixer"].params for blk in b.blocks]
    left = a.blocks[1].children["mixer"].children["left"]
    assert left.params["window"] == 33 and left.params["keep_first"] == 5


def test_parts_refuse_what_their_kernels_do_not_take():
    from pytorch_transformers_b200 import kernels
    from pytorch_transformers_b200.parts.base import BuildContext, PartSpec, make_part
    build = BuildContext(torch.device("cpu"), torch.float32, kernels)
    d = {"hidden": 8, "heads": 2, "kv_heads": 1, "dim": 8, "vdim": 8, "taps": 3}
    for bad in (dict(dim=300), dict(taps=0), dict(taps=70), dict(kv_heads=3), dict(decay="row"), dict(gate="wide"), dict(gate_act="relu")):
        with pytest.raises(ValueError):
            make_part(build, PartSpec("mixer", "delta_rule", dict(d, **bad)))
    ex = {"hidden": 8, "inner": 8, "experts": 4, "top": 2}
    for bad in (dict(expert="clamped_glu"), dict(expert="clamped_glu", limit=-1.0), dict(limit=2.0), dict(expert="clamped_glu", limit=1.0, weight_on="input")):
        with pytest.raises(ValueError):
            make_part(build, PartSpec("feed_forward", "routed_experts", dict(ex, **bad)))
    norm = PartSpec("norm", "layernorm", {"size": 8, "eps": 1e-5})
    with pytest.raises(ValueError):
        make_part(build, PartSpec("block", "post_norm", children={"mixer": PartSpec("mixer", "delta_rule", d), "norm_mixer": norm}))
    with pytest.raises(ValueError):
        make_part(build, PartSpec("token_input", "gated_table", {"hidden": 8, "dim": 0, "first": 0, "eps": 1e-5}))


def test_frequency_bands_of_the_position_part():
    from pytorch_transformers_b200.parts.position import banded_frequencies
    sc = {"factor": 5.0, "low": 1.25, "high": 6.0, "original": 300}
    got = banded_frequencies(36, 2000.0, **sc)
    torch.testing.assert_close(got, torch.tensor(plain.frequencies({"dims": 36, "base": 2000.0, "scaling": sc}), dtype=F64), atol=0, rtol=1e-14)


# ------------------------------------------------------------------------------------------------ the oracle with itself
def _rule(T, H, d, dv, seed):
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    return (plain.unit(rn(T, H, d)), plain.unit(rn(T, H, d)), rn(T, H, dv), torch.rand(T, H, d, generator=g, dtype=F64),
            torch.rand(T, H, generator=g, dtype=F64))


def test_plain_rule_in_two_halves_and_as_linear_equations():
    T, H, d, dv = 11, 2, 5, 4
    q, k, v, a, b = _rule(T, H, d, dv, 1)
    whole, S = plain.delta_recurrence(q, k, v, a, b)
    one, S1 = plain.delta_recurrence(q[:6], k[:6], v[:6], a[:6], b[:6])
    two, S2 = plain.delta_recurrence(q[6:], k[6:], v[6:], a[6:], b[6:], S1)
    torch.testing.assert_close(torch.cat([one, two]), whole)
    torch.testing.assert_close(S2, S)
    for h in range(H):      # u solves (I + diag(b) strictly-lower (k decayed k)) u = diag(b) v; o = lower (q decayed k) u
        A, P = torch.zeros(T, T, dtype=F64), torch.zeros(T, T, dtype=F64)
        for t in range(T):
            for s in range(t + 1):
                fade = a[s + 1:t + 1, h].prod(0)
                A[t, s], P[t, s] = (k[t, h] * k[s, h] * fade).sum(), (q[t, h] * k[s, h] * fade).sum()
        u = torch.linalg.solve(torch.eye(T, dtype=F64) + b[:, h:h + 1] * A.tril(-1), b[:, h:h + 1] * v[:, h])
        torch.testing.assert_close(P @ u, whole[:, h])


def test_plain_rule_writes_over_what_the_same_key_held():
    q, k, v, a, b = _rule(6, 1, 4, 3, 2)
    k[4], b[4], a[:] = k[1], 1.0, 1.0
    q[5] = k[1]
    k[5], b[5] = plain.unit(k[5] - (k[5] * k[1]).sum() * k[1]), 1.0
    o, _ = plain.delta_recurrence(q, k, v, a, b)
    torch.testing.assert_close(o[5], v[4], atol=1e-5, rtol=1e-5)      # the root's 1e-6 keeps the keys short of length one


def test_plain_convolution_window_and_unit_vectors():
    x = torch.arange(1.0, 6.0, dtype=F64)[:, None]
    y = plain.short_conv(x, torch.tensor([[100.0, 10.0, 1.0]], dtype=F64))
    assert y.flatten().tolist() == [1.0, 12.0, 123.0, 234.0, 345.0]
    assert plain.short_conv(x[:1], torch.tensor([[100.0, 10.0, 1.0]], dtype=F64)).flatten().tolist() == [1.0]
    z = torch.tensor([[3.0, 4.0], [0.0, 0.0]], dtype=F64)
    torch.testing.assert_close(plain.unit(z), torch.tensor([[0.6, 0.8], [0.0, 0.0]], dtype=F64), atol=1e-7, rtol=0)


def test_plain_decays_lie_between_zero_and_one_and_spread_over_channels():
    g = torch.Generator().manual_seed(3)
    rn = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    h, m = rn(5, 6), {"heads": 2, "dim": 3}
    per_head = plain.delta_decay(h, {"a": rn(2, 6), "dt_bias": rn(2), "A_log": rn(2)}, m)
    assert per_head.shape == (5, 2, 3) and torch.equal(per_head[..., 0], per_head[..., 2])
    per_channel = plain.delta_decay(h, {"a1": rn(2, 6), "a2": rn(6, 2), "dt_bias": rn(6), "A_log": rn(2)}, m)
    assert per_channel.shape == (5, 2, 3) and not torch.equal(per_channel[..., 0], per_channel[..., 2])
    assert float(per_channel.min()) > 0 and float(per_channel.max()) < 1


def test_plain_frequencies_keep_mix_and_divide():
    sc = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 100.0}
    rot = {"dims": 16, "base": 100.0, "scaling": sc}
    got, base = plain.frequencies(rot), plain.frequencies({"dims": 16, "base": 100.0})
    for f, b in zip(got, base):
        wave = 2 * math.pi / b
        if wave < 25:
            assert f == b
        elif wave > 100:
            assert f == b / 4
        else:
            assert b / 4 < f < b
    assert got[0] == base[0] and got[-1] == base[-1] / 4


def test_plain_window_and_added_one():
    vis = plain.visible(10, {"size": 3, "keep_first": 2})
    assert vis[9].tolist() == [True, True, False, False, False, False, False, True, True, True]
    assert plain.visible(4, {"size": 1}).int().tolist() == torch.eye(4).int().tolist()
    assert plain.visible(3, None).int().tolist() == [[1, 0, 0], [1, 1, 0], [1, 1, 1]]
    s = torch.randn(1, 6, dtype=F64) * 3
    p = plain.sink_softmax(s, torch.ones(1, 6, dtype=torch.bool))
    torch.testing.assert_close(p[0], torch.softmax(torch.cat([s[0], torch.zeros(1, dtype=F64)]), 0)[:-1])


def test_plain_router_weighs_without_the_correction():
    g = torch.Generator().manual_seed(7)
    h, w, c = torch.randn(30, 6, generator=g, dtype=F64), torch.randn(5, 6, generator=g, dtype=F64), torch.randn(5, generator=g, dtype=F64)
    ids, weights = plain.route(h, w, c, 2)
    s = torch.softmax(h @ w.T, -1)
    for t in range(30):
        assert set(ids[t].tolist()) == set(sorted(range(5), key=lambda e: -float(s[t, e] + c[e]))[:2])
        torch.testing.assert_close(weights[t], s[t, ids[t]])
        assert float(weights[t].sum()) < 1
