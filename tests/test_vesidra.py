"""Vesidra without a GPU: configuration and registry, the spec (tensor names and shapes, one cache row per token and
layer), refused configurations and parts, and the plain implementation's own consistency (a latent attention with the key
up-projection folded into the query, the scaled frequencies against their definition and against the library's table, the
router's weights, the shared expert)."""
import json
import math

import pytest
import torch

import plain_vesidra as plain
import vesidra_models as vm

F64 = torch.float64


def test_registry_finds_the_design_by_its_architecture_string(tmp_path):
    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200.config.registry import lookup
    folder = vm.write_folder(tmp_path, "mixed")
    cfg = ptb.AutoConfig.from_pretrained(folder)
    assert isinstance(cfg, ptb.VesidraConfig) and cfg.vocab == 203 and cfg.width == 88 and len(cfg.layers) == 4
    assert cfg.vocab_size == 203 and cfg.hidden_size == 88 and cfg.num_hidden_layers == 4 and cfg.tie_word_embeddings
    assert lookup({"architecture": "Vesidra"}).model_type == "vesidra"
    back = ptb.VesidraConfig.from_dict(json.loads(json.dumps(cfg.to_dict())))
    assert back.layers == cfg.layers and back.norm == cfg.norm and back.embedding == cfg.embedding


@pytest.mark.parametrize("name", sorted(vm.CONFIGS))
def test_spec_names_every_tensor_and_states_every_need(name):
    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200.models.vesidra import vesidra_spec
    raw = vm.CONFIGS[name]
    cfg = ptb.VesidraConfig.from_dict(raw)
    spec = vesidra_spec(cfg)
    assert spec.stream_float32 and spec.head_name is None and spec.embedding_norm is None
    assert spec.embedding_scale == raw["embedding"]["scale"]
    model = ptb.CausalLM(spec, cfg, device="cpu", dtype=torch.float32)
    table, want = model.param_table(), vm.tensor_shapes(raw)
    assert set(table) == set(want)
    for tensor, (_, _, decl) in table.items():
        assert tuple(decl.shape) == tuple(want[tensor]), tensor
    for (entry, c, s), layer in zip(model.cache_needs(), raw["layers"]):
        m = layer["mixer"]
        # one row per token for all heads: the latent and the rotated key part; no value rows, no state
        assert s is None and (c.kind, c.kv_heads, c.head_dim, c.v_head_dim) == ("full", 1, m["kv_rank"] + m["rot_dim"], 0)
    assert model.use_graphs and len(model.blocks) == len(raw["layers"])


def _with(name, **changes):
    cfg = json.loads(json.dumps(vm.CONFIGS[name]))
    for path, value in changes.items():
        at = cfg
        keys = path.split("__")
        for k in keys[:-1]:
            at = at[int(k)] if k.isdigit() else at[k]
        at[int(keys[-1]) if keys[-1].isdigit() else keys[-1]] = value
    return cfg


@pytest.mark.parametrize("bad", [
    dict(vocab=0), dict(width=-1), dict(layers=[]), dict(norm={"eps": 0}), dict(embedding={"scale": 0}), dict(layers__0__type="gla"),
    dict(layers__0__mixer__heads=0), dict(layers__0__mixer__kv_rank=None), dict(layers__0__mixer__rot_dim=7),
    dict(layers__0__mixer__rot_dim=0), dict(layers__0__mixer__scale=0), dict(layers__0__mixer__rot=None),
    dict(layers__0__mixer__rot__base=0), dict(layers__0__mixer__rot__dims=16), dict(layers__0__mixer__rot__scaling__factor=0),
    dict(layers__0__mixer__rot__scaling={"factor": 2.0}), dict(layers__0__mlp__router__top=8), dict(layers__0__mlp__expert={}),
    dict(layers__0__mlp__shared={"ff": 0}), dict(layers__1__mlp={"kind": "dense"}), dict(layers__1__mlp={"kind": "glu", "ff": 8}),
])
def test_configurations_that_cannot_be_built_are_refused(bad):
    import pytorch_transformers_b200 as ptb
    with pytest.raises(ptb.ConfigError):
        ptb.VesidraConfig.from_dict(_with("mixed", **bad))


def test_optional_keys():
    """No ``rot.dims`` (it is rot_dim), no scaling, ``shared`` null, a layer without ``mlp``, keys the design does not know."""
    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200.models.vesidra import vesidra_spec
    raw = _with("mixed", layers__0__mlp__shared=None, layers__0__mixer__note="x", layers__0__mixer__rot={"base": 10.0}, seed=3)
    del raw["layers"][1]["mlp"]
    spec = vesidra_spec(ptb.VesidraConfig.from_dict(raw))
    assert "shared" not in spec.blocks[0].children["feed_forward"].children and "feed_forward" not in spec.blocks[1].children
    rotary = spec.blocks[0].children["mixer"].children["position"].params
    assert rotary["rotary_dim"] == 24 and "yarn" not in rotary


def test_parts_refuse_what_their_kernels_do_not_take():
    from pytorch_transformers_b200 import kernels
    from pytorch_transformers_b200.parts.base import BuildContext, PartSpec, make_part
    build = BuildContext(torch.device("cpu"), torch.float32, kernels)
    m = {"hidden": 8, "heads": 2, "dim": 8, "rot_dim": 4, "vdim": 8, "q_rank": None, "kv_rank": 16, "scale": 1.0, "eps": 1e-5}
    for bad in (dict(gate="layer"), dict(kv_rank=513), dict(q_rank=0), dict(heads=0), dict(rot_dim=-2)):
        with pytest.raises(ValueError):
            make_part(build, PartSpec("mixer", "latent_attention", dict(m, **bad)))
    ex = {"hidden": 8, "inner": 8, "experts": 4, "top": 2}
    for bad in (dict(score="logits"), dict(score="softmax_chosen", normalize=True), dict(weight_on="input"),
                dict(expert="plain", activation="cube"), dict(top=5)):
        with pytest.raises(ValueError):
            make_part(build, PartSpec("feed_forward", "routed_experts", dict(ex, **bad)))
    with pytest.raises(ValueError):
        make_part(build, PartSpec("feed_forward", "dense", {"hidden": 8, "inner": 8, "bias": True, "wide_out": True}))


def test_projections_of_the_input_are_one_matrix_in_whole_words():
    """Queries, latent and gates are rows of one matrix; its row count is brought to a multiple of 8 with rows of zeros."""
    from pytorch_transformers_b200 import kernels
    from pytorch_transformers_b200.parts.base import BuildContext, PartSpec, make_part
    part = make_part(BuildContext(torch.device("cpu"), torch.float32, kernels), PartSpec(
        "mixer", "latent_attention", {"hidden": 12, "heads": 3, "dim": 5, "rot_dim": 2, "vdim": 4, "q_rank": None, "kv_rank": 6,
                                      "scale": 1.0, "eps": 1e-5, "gate": "head"}))
    g = torch.Generator().manual_seed(0)
    t = {n: torch.randn(d.shape, generator=g) for n, d in part.param_decls().items()}
    assert t["g"].shape == (3, 12) and "dq" not in t
    part.bind(t)
    rows = 21 + 8 + 3
    assert part.p_in.shape == (rows, 12)
    torch.testing.assert_close(part.p_in, torch.cat([t["q"], t["dkv"], t["g"]]))
    t["g"] = torch.randn(1, 12, generator=g)        # 30 rows: two rows of zeros follow
    part.bind(t)
    assert part.p_in.shape == (32, 12) and float(part.p_in[30:].abs().max()) == 0.0 and float(part.p_in[29].abs().max()) > 0


# ------------------------------------------------------------------------------------------------ the plain implementation
def test_plain_scaled_frequencies():
    rot = {"dims": 32, "base": 10000.0, "scaling": {"factor": 8.0, "original": 512, "fast": 16.0, "slow": 1.0}}
    f, mult = plain.frequencies(rot)
    raw = [10000.0 ** (-2 * i / 32) for i in range(16)]
    turns = [512 * r / (2 * math.pi) for r in raw]          # turns of each pair over the original context
    assert math.isclose(mult, 0.1 * math.log(8.0) + 1.0)
    assert all(math.isclose(a, b) for a, b, t in zip(f, raw, turns) if t > 32)              # fast pairs stay
    assert all(math.isclose(a, b / 8) for a, b, t in zip(f, raw, turns) if t < 0.5)         # slow pairs are divided
    assert any(b / 8 * 1.01 < a < b * 0.99 for a, b in zip(f, raw))                         # and a ramp lies between
    assert plain.frequencies({"dims": 8, "base": 7.0}) == ([7.0 ** (-i / 4) for i in range(4)], 1.0)


@pytest.mark.parametrize("yarn", [(4.0, 60, 8.0, 1.0), (16.0, 4096, 32.0, 1.0), (1.0, 1, 1.0, 1.0), (3.0, 77, 5.0, 0.5), (2.0, 10, 9.0, 8.0)])
@pytest.mark.parametrize("dims,base", [(2, 100.0), (24, 20000.0), (64, 1e6)])
def test_the_librarys_table_of_scaled_frequencies(dims, base, yarn):
    from pytorch_transformers_b200.parts.position import yarn_frequencies
    sc = dict(zip(("factor", "original", "fast", "slow"), yarn))
    f, mult = yarn_frequencies(dims, base, **{k: float(v) for k, v in sc.items()})
    want, want_mult = plain.frequencies({"dims": dims, "base": base, "scaling": sc})
    torch.testing.assert_close(f, torch.tensor(want, dtype=F64), rtol=1e-12, atol=0)
    assert math.isclose(mult, want_mult)


def test_plain_rotation_turns_pairs_half_the_size_apart():
    g = torch.Generator().manual_seed(1)
    rot = {"dims": 6, "base": 50.0}
    x = torch.randn(4, 2, 6, generator=g, dtype=F64)
    pos = torch.tensor([0, 1, 5, 40])
    y = plain.rotate(x, pos, rot)
    torch.testing.assert_close(y[0], x[0])
    z = torch.complex(x[..., :3], x[..., 3:]) * torch.exp(1j * pos[:, None, None] * torch.tensor(plain.frequencies(rot)[0], dtype=F64))
    torch.testing.assert_close(y, torch.cat([z.real, z.imag], -1))


def test_plain_attention_with_the_key_projection_folded_into_the_query():
    g = torch.Generator().manual_seed(2)
    m = {"heads": 2, "dim": 5, "rot_dim": 4, "vdim": 3, "kv_rank": 7, "scale": 0.4, "rot": {"base": 30.0, "dims": 4}}
    rn = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    w = {"uk": rn(10, 7), "uv": rn(6, 7)}
    q, c, kr = rn(9, 2, 9), rn(9, 7), rn(9, 4)
    got = plain.latent_heads(q, c, kr, w, m)
    for h in range(2):
        folded = q[:, h, :5] @ w["uk"].reshape(2, 5, 7)[h]
        p = plain.causal_softmax((folded @ c.T + q[:, h, 5:] @ kr.T) * 0.4)
        torch.testing.assert_close((p @ c) @ w["uv"].reshape(2, 3, 7)[h].T, got[:, h])
    # rows from the middle of a sequence on
    torch.testing.assert_close(plain.latent_heads(q[6:], c, kr, w, m, first_query=6), got[6:])


def test_plain_router_and_mixture():
    g = torch.Generator().manual_seed(3)
    rn = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    h, wr, b = rn(40, 10), rn(6, 10), 2 * rn(6)
    ids, weights = plain.route(h, wr, b, 3)
    z = h @ wr.T + b
    for t in range(40):
        assert sorted(ids[t].tolist()) == sorted(sorted(range(6), key=lambda e: -float(z[t, e]))[:3])
        torch.testing.assert_close(weights[t], torch.softmax(z[t, ids[t]], 0))
    w = {f"e{e}.{n}": rn(*s) for e in range(6) for n, s in (("up", (4, 10)), ("down", (10, 4)))}
    w.update({"router": wr, "router.b": b, "shared.up": rn(5, 10), "shared.down": rn(10, 5)})
    mlp = {"kind": "moe", "router": {"experts": 6, "top": 6}, "expert": {"ff": 4}, "shared": {"ff": 5}}
    every = sum(torch.softmax(z, -1)[:, e:e + 1] * (torch.relu(h @ w[f"e{e}.up"].T).square() @ w[f"e{e}.down"].T) for e in range(6))
    torch.testing.assert_close(plain.moe_ff(h, w, mlp), every + torch.relu(h @ w["shared.up"].T).square() @ w["shared.down"].T)
