"""Random Vesidra configurations under random cuttings of the work, against the plain implementation.

The fixed configurations of tests/vesidra_models.py pin known corners; this draws others: widths, head counts, plain,
rotated, value and latent sizes (also those of the tensor-core kernels, ones beyond them and ones that are no multiple of
8), rotations with and without scaling whose ramp covers all, some and none of the pairs, dense and routed feed-forwards
and none, with and without a shared expert, in float32 and bfloat16. Every request is fed as a prompt of a random length
(in one step, or in two or three portions), then token by token in a batch whose members end at different times, and
every logit row is compared.
"""
import os
import random

import numpy as np
import pytest
import torch

import plain_vesidra as plain
import tiny_models as tm
import vesidra_models as vm

pytestmark = pytest.mark.gpu


def random_mlp(r: random.Random):
    kind = r.choice(["none", "dense", "dense", "moe", "moe", "moe"])
    if kind == "none":
        return None
    if kind == "dense":
        return vm.dense(r.choice([24, 56, 200]))
    experts = r.choice([1, 2, 3, 5, 8, 16])
    return vm.moe(experts, r.randint(1, min(experts, 6)), r.choice([16, 40, 72]), shared=r.choice([None, 8, 48, 100]))


def random_mixer(r: random.Random):
    dim, rot, vdim = r.choice([(8, 8, 8), (12, 4, 20), (24, 8, 12), (48, 16, 64), (40, 24, 40), (64, 32, 64), (96, 32, 128),
                               (128, 64, 128), (100, 60, 90), (64, 64, 32), (30, 2, 17), (160, 40, 64), (56, 48, 150), (1, 2, 3)])
    rank = r.choice([5, 12, 16, 32, 48, 64, 80, 100, 112, 128, 192, 200])
    yarn = r.choice([None, (4.0, 64, 8.0, 1.0), (8.0, 1024, 32.0, 1.0), (1.0, 100, 4.0, 2.0), (40.0, 33, 30.0, 0.5), (2.0, 8192, 64.0, 0.25)])
    return vm.mla(r.choice([1, 2, 3, 5, 8, 17]), dim, rot, vdim, rank, r.choice([(dim + rot) ** -0.5, 0.3, 0.1, 1.0 / (dim + rot)]),
                  r.choice([10.0, 500.0, 10000.0, 1e6]), yarn)


def random_config(r: random.Random) -> dict:
    layers = [dict(random_mixer(r), mlp=random_mlp(r)) for _ in range(r.choice([1, 2, 3, 4, 5]))]
    return {"architecture": "Vesidra", "vocab": r.choice([61, 200, 515]), "width": r.choice([40, 64, 72, 136, 256]),
            "embedding": {"scale": r.choice([1.0, 0.3, 5.5, 16.0])}, "norm": {"eps": r.choice([1e-5, 1e-6, 1e-3])}, "layers": layers}


def row_errors(got, ref):
    got, ref = got.double().cpu().reshape(-1, got.shape[-1]), ref.double().cpu().reshape(-1, ref.shape[-1])
    return (got - ref).norm(dim=1) / ref.norm(dim=1).clamp_min(1e-30)


@pytest.mark.parametrize("first_seed", range(0, 48, 8))
def test_random_configurations_and_cuttings(tmp_path, first_seed):
    import pytorch_transformers_b200 as ptb
    for seed in range(first_seed, first_seed + 8):
        r = random.Random(17000 + seed)
        cfg = random_config(r)
        dtype = r.choice(["float32", "float32", "bfloat16"])
        if dtype == "bfloat16":
            cfg = vm.steady(cfg)        # no choice of experts within a bfloat16 rounding of another
        folder = tm.write_model_folder(os.path.join(str(tmp_path), f"m{seed}"), cfg, vm.make_weights(cfg, seed),
                                       bf16=(dtype == "bfloat16"))
        model = ptb.AutoModelForCausalLM.from_pretrained(folder, dtype=dtype)
        w = vm.torch_weights(cfg, seed)
        g = np.random.Generator(np.random.PCG64(seed))
        lengths = [int(g.integers(2, r.choice([40, 150, 400]))) for _ in range(r.choice([1, 2, 3, 5]))]
        reqs = [g.integers(0, cfg["vocab"], size=n).tolist() for n in lengths]
        refs = [plain.forward(cfg, w, q) for q in reqs]
        what = f"seed {seed} {dtype} {cfg}"
        errors = []

        def compare(got, want):
            errors.append(row_errors(got, want))

        cache = model.new_cache(sum((n + 63) // 64 * 64 for n in lengths) + 64)
        slots = [cache.open() for _ in reqs]
        heads = [int(g.integers(1, n + 1)) for n in lengths]
        cuts = r.choice([1, 2, 3])
        marks = [sorted({0, h} | {int(g.integers(1, h + 1)) for _ in range(cuts - 1)}) for h in heads]
        for step in range(cuts):
            part = [(i, marks[i][step], marks[i][step + 1]) for i in range(len(reqs)) if step + 1 < len(marks[i])]
            if not part:
                break
            out, at = model.step(cache, [slots[i] for i, _, _ in part], [reqs[i][a:b] for i, a, b in part], want="all"), 0
            for i, a, b in part:
                compare(out[at:at + b - a], refs[i][a:b])
                at += b - a
        pos = list(heads)
        for i in [i for i in range(len(reqs)) if pos[i] >= lengths[i]]:
            cache.close(slots[i])
        live = [i for i in range(len(reqs)) if pos[i] < lengths[i]]
        for _ in range(80):
            if not live:
                break
            out = model.step(cache, [slots[i] for i in live], [[reqs[i][pos[i]]] for i in live], want="last")
            for row, i in enumerate(live):
                compare(out[row:row + 1], refs[i][pos[i]:pos[i] + 1])
                pos[i] += 1
            for i in [i for i in live if pos[i] >= lengths[i]]:
                cache.close(slots[i])
            live = [i for i in live if pos[i] < lengths[i]]
        model.check_errors()
        cache.check()
        e = torch.cat(errors)
        if dtype == "float32":
            assert e.max() < 2e-4 and e.median() < 2e-5, f"{what}: worst row error {e.max():.3g}, median {e.median():.3g}"
        else:
            assert e.median() < 3e-2 and (e < 6e-2).double().mean() >= 0.9, \
                f"{what}: median row error {e.median():.3g}, worst {e.max():.3g}"
