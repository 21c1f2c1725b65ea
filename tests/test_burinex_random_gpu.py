"""Burinex configurations drawn at random (layer order, sizes, head counts, windows, rotations, decays, experts, constants), each
with random weights, in float32 against the plain implementation and in bfloat16 against what rounding alone does: a whole prompt,
most of it in one step and the rest token by token, and two unequal requests in one batch that decode together."""
import random

import pytest
import torch

import plain_burinex as plain
from conftest import rel_err

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def draw_config(seed):
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(1, 5)):
        kind = rng.choice(["attention", "latent_attention", "lightning"])
        heads, dim = rng.choice([1, 2, 3, 6]), rng.choice([5, 8, 16, 24, 64, 80, 128])
        m = {"heads": heads, "dim": dim, "vdim": rng.choice([dim, 7, 16, 40, 96])}
        if kind == "attention":
            m["kv_heads"] = rng.choice([d for d in range(1, heads + 1) if heads % d == 0])
            m["scale"] = rng.uniform(0.5, 1.5) * dim ** -0.5
            if rng.random() < 0.8:
                m["q_temp"] = {"coef": rng.choice([-0.1, 0.1, 0.6]), "every": rng.choice([1, 9, 64, 100])}
        elif kind == "latent_attention":
            m.update(rot_dim=rng.choice([0, 2, 8, 32, 64]), kv_rank=rng.choice([6, 16, 40, 64, 72, 128, 264]), q_rank=rng.choice([5, 24, 64]))
            m["scale"] = rng.uniform(0.5, 1.5) * (dim + m["rot_dim"]) ** -0.5
            if rng.random() < 0.8:
                m["mask"] = {"size": rng.choice([1, 3, 33, 64, 100, 128, 400])}
            if m["rot_dim"]:
                m["rot"] = {"base": rng.choice([30.0, 5000.0, 1e6]), "dims": rng.choice([m["rot_dim"], m["rot_dim"] // 2 // 2 * 2])}
                if rng.random() < 0.7:
                    m["rot"]["scaling"] = {"factor": rng.choice([1.0, 2.0, 40.0]), "original": rng.choice([16, 200, 4096]),
                                           "fast": rng.choice([4.0, 32.0]), "slow": rng.choice([0.5, 1.0])}
        else:
            m["decay"] = [rng.choice([0.1, 0.6, 0.9, 0.99, 0.9999]) for _ in range(heads)]
        mlp = None
        if rng.random() < 0.7:
            experts = rng.choice([1, 2, 5, 16, 33])
            mlp = {"kind": "moe", "router": {"experts": experts, "top": rng.randint(1, min(experts, 4))}, "expert": {"ff": rng.choice([7, 16, 40])}}
            if rng.random() < 0.7:
                mlp["shared"] = {"ff": rng.choice([5, 32, 64])}
        layers.append({"type": kind, "mixer": m, "mlp": mlp})
    cfg = {"architecture": "Burinex", "vocab": rng.randint(40, 300), "width": rng.choice([22, 40, 52, 64, 96, 136]),
           "norm": {"eps": rng.choice([1e-6, 1e-5, 1e-2])}, "postln_alpha": rng.uniform(0.7, 4.0), "layers": layers}
    if rng.random() < 0.8:
        cfg["logit_softcap"] = rng.uniform(3.0, 40.0)
    return cfg


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(24))
def test_a_configuration_drawn_at_random(pe, seed, dtype):
    cfg = draw_config(1000 + seed)
    w = plain.random_weights(cfg, 2000 + seed)
    eng = pe.Engine(None, config=pe.BurinexConfig.from_dict(cfg), weights={k: v.to(DEV) for k, v in w.items()}, dtype=dtype,
                    max_context_len=512, max_cache_tokens=64 * 24, max_batch=4)
    g = torch.Generator().manual_seed(seed)
    long = torch.randint(0, cfg["vocab"], (150,), generator=g).tolist()
    short = torch.randint(0, cfg["vocab"], (37,), generator=g).tolist()
    ref_long, ref_short = plain.forward(cfg, w, long), plain.forward(cfg, w, short)
    with plain.stored(torch.bfloat16):
        noise_long = (plain.forward(cfg, w, long) - ref_long).pow(2).mean(1).sqrt()
        noise_short = (plain.forward(cfg, w, short) - ref_short).pow(2).mean(1).sqrt()

    def check(got, ref, noise, what):
        got = got.double().cpu()
        if dtype == "float32":
            assert rel_err(got, ref) < 3e-5, (seed, what, cfg)
        else:                     # the median: a rounding may pick another expert here and there
            limit = 4.0 * max(float(noise.median()), float(noise_long.median()))
            assert float((got - ref).pow(2).mean(1).sqrt().median()) < limit, (seed, what, cfg)

    s = eng.alloc_slot()
    check(eng.step([pe.StepEntry(s, long, tuple(range(150)))]).clone(), ref_long, noise_long, "whole")
    eng.free_slot(s)
    s = eng.alloc_slot()
    rows = [eng.step([pe.StepEntry(s, long[:110], (109,))]).clone()]
    for t in long[110:]:
        rows.append(eng.step([pe.StepEntry(s, [t], (0,))]).clone())
    eng.free_slot(s)
    check(torch.cat(rows), ref_long[109:], noise_long[109:], "decoded")
    # two unequal requests start together, decode together, the shorter one ends earlier
    a, b = eng.alloc_slot(), eng.alloc_slot()
    out = eng.step([pe.StepEntry(a, long[:120], (119,)), pe.StepEntry(b, short[:30], (29,))]).clone()
    got_a, got_b = [out[0:1]], [out[1:2]]
    for i in range(12):
        entries = [pe.StepEntry(a, [long[120 + i]], (0,))]
        if 30 + i < len(short):
            entries.append(pe.StepEntry(b, [short[30 + i]], (0,)))
        out = eng.step(entries).clone()
        got_a.append(out[0:1])
        if len(entries) == 2:
            got_b.append(out[1:2])
            if 30 + i == len(short) - 1:
                eng.free_slot(b)
    eng.free_slot(a)
    check(torch.cat(got_a), ref_long[119:132], noise_long[119:132], "together, long")
    check(torch.cat(got_b), ref_short[29:37], noise_short[29:37], "together, short")
    assert not eng.cache.live_slots
    eng.cache.check()
