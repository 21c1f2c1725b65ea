"""Bobasun configurations drawn at random (sizes, head counts, streams, rotations, value mixing, constants), each with random
weights, in float32 against the plain implementation and in bfloat16 against what rounding alone does: a whole prompt, most of
it in one step and the rest token by token, and two unequal requests in one batch that decode together."""
import random

import pytest
import torch

import plain_bobasun as plain
from conftest import rel_err

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def _divisor(rng, n):
    return rng.choice([d for d in range(1, n + 1) if n % d == 0])


def draw_config(seed):
    rng = random.Random(seed)
    layers = []
    shared = (rng.choice([1, 2, 3]), rng.choice([6, 8, 16, 40, 64, 100, 128]))     # kv heads and value size of the mixing layers
    for _ in range(rng.randint(1, 5)):
        mix = rng.random() < 0.6
        kv = shared[0] if mix else rng.choice([1, 2, 3])
        dim = rng.choice([5, 8, 12, 16, 24, 64, 80, 128, 136])
        m = {"heads": kv * rng.choice([1, 2, 3, 5]), "kv_heads": kv, "dim": dim, "vdim": shared[1] if mix else rng.choice([dim, 8, 20, 72]),
             "scale": rng.uniform(0.3, 2.0) * dim ** -0.5, "v_mix": mix}
        dims = rng.choice([0, 2, dim // 2 // 2 * 2, dim // 2 * 2])
        if dims:
            m["rot"] = {"base": rng.choice([30.0, 5000.0, 1e6]), "dims": dims}
            if rng.random() < 0.7:
                m["rot"]["scaling"] = {"factor": rng.choice([1.0, 1.5, 8.0, 40.0])}
        mlp = None if rng.random() < 0.2 else {"kind": "dense", "ff": rng.choice([7, 24, 64, 128, 136]), "limit": rng.uniform(0.3, 5.0)}
        layers.append({"type": "attention", "mixer": m, "mlp": mlp})
    cfg = {"architecture": "Bobasun", "vocab": rng.randint(40, 300), "width": rng.choice([22, 40, 52, 64, 96, 136]),
           "streams": rng.choice([1, 2, 3, 4, 5, 7, 10]), "norm": {"eps": rng.choice([1e-6, 1e-5, 1e-2])}, "layers": layers}
    if rng.random() < 0.7:
        cfg["embedding"] = {"scale": rng.uniform(0.5, 12.0)}
    return cfg


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(20))
def test_a_configuration_drawn_at_random(pe, seed, dtype):
    cfg = draw_config(1000 + seed)
    w = plain.random_weights(cfg, 2000 + seed)
    eng = pe.Engine(None, config=pe.BobasunConfig.from_dict(cfg), weights={k: v.to(DEV) for k, v in w.items()}, dtype=dtype,
                    max_context_len=512, max_cache_tokens=64 * 24, max_batch=4)
    g = torch.Generator().manual_seed(seed)
    long = torch.randint(0, cfg["vocab"], (150,), generator=g).tolist()
    short = torch.randint(0, cfg["vocab"], (37,), generator=g).tolist()
    ref_long, ref_short = plain.forward(cfg, w, long), plain.forward(cfg, w, short)
    with plain.stored(torch.bfloat16):
        noise = float((plain.forward(cfg, w, long) - ref_long).pow(2).mean(1).sqrt().mean())

    def check(got, ref, what):
        got = got.double().cpu()
        if dtype == "float32":
            assert rel_err(got, ref) < 3e-5, (seed, what, cfg)
        else:
            assert float((got - ref).pow(2).mean(1).sqrt().mean()) < 2.5 * noise, (seed, what, cfg)

    s = eng.alloc_slot()
    check(eng.step([pe.StepEntry(s, long, tuple(range(150)))]).clone(), ref_long, "whole")
    eng.free_slot(s)
    s = eng.alloc_slot()
    rows = [eng.step([pe.StepEntry(s, long[:110], (109,))]).clone()]
    for t in long[110:]:
        rows.append(eng.step([pe.StepEntry(s, [t], (0,))]).clone())
    eng.free_slot(s)
    check(torch.cat(rows), ref_long[109:], "decoded")
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
    check(torch.cat(got_a), ref_long[119:132], "together, long")
    check(torch.cat(got_b), ref_short[29:37], "together, short")
    assert not eng.cache.live_slots
    eng.cache.check()
