"""What needs no GPU of the Burinex architecture: its configuration file, its plan (tensor names, cache entries), rotary tables with
scaled frequencies, and the plain implementation's own consistency."""
import copy
import math
from importlib import import_module

import pytest
import torch

import plain_burinex as plain

CFG = {"architecture": "Burinex", "vocab": 71, "width": 36, "norm": {"eps": 1e-4}, "postln_alpha": 1.4, "logit_softcap": 6.0,
       "layers": [
           {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 10, "vdim": 6, "scale": 0.4, "q_temp": {"coef": 0.5, "every": 7}},
            "mlp": {"kind": "moe", "router": {"experts": 5, "top": 2}, "expert": {"ff": 12}, "shared": {"ff": 20}}},
           {"type": "latent_attention", "mixer": {"heads": 3, "dim": 8, "rot_dim": 6, "vdim": 10, "kv_rank": 14, "q_rank": 16, "scale": 0.3,
                                                  "mask": {"size": 9},
                                                  "rot": {"base": 50.0, "dims": 6, "scaling": {"factor": 3.0, "original": 32, "fast": 4.0, "slow": 1.0}}},
            "mlp": None},
           {"type": "lightning", "mixer": {"heads": 2, "dim": 6, "vdim": 8, "decay": [0.6, 0.98]},
            "mlp": {"kind": "moe", "router": {"experts": 3, "top": 1}, "expert": {"ff": 8}}},
           {"type": "latent_attention", "mixer": {"heads": 2, "dim": 6, "rot_dim": 8, "vdim": 4, "kv_rank": 10, "q_rank": 12, "scale": 0.5,
                                                  "rot": {"base": 90.0, "dims": 4}},
            "mlp": {"kind": "moe", "router": {"experts": 2, "top": 2}, "expert": {"ff": 6}, "shared": {"ff": 4}}}]}


def test_config_reads_every_layer_by_itself_and_writes_it_back(pe):
    cfg = pe.BurinexConfig.from_dict(CFG)
    assert (cfg.postln_alpha, cfg.logit_softcap, cfg.norm_eps, cfg.vocab_size) == (1.4, 6.0, 1e-4, 71)
    assert cfg.layers[1].mixer.window == 9 and cfg.layers[3].mixer.window is None and cfg.layers[1].mlp is None
    assert cfg.layers[2].mixer.decay == (0.6, 0.98) and cfg.layers[2].mlp.shared_ff == 0
    assert cfg.to_dict() == CFG and pe.BurinexConfig.from_dict(cfg.to_dict()) == cfg
    assert pe.config.architecture_of(CFG).name == "Burinex"
    for path, value, word in [(("layers", 0, "type"), "delta", "type"), (("layers", 0, "mixer", "kv_heads"), 3, "multiple"),
                              (("layers", 1, "mixer", "rot", "dims"), 8, "dims"), (("layers", 1, "mixer", "rot", "dims"), 5, "even"),
                              (("layers", 0, "mlp", "kind"), "dense", "kind"), (("layers", 0, "mlp", "router", "top"), 6, "top"),
                              (("layers", 2, "mixer", "decay"), [0.5], "decay"), (("layers", 2, "mixer", "decay"), [0.5, 1.5], "decay"),
                              (("norm",), None, "norm"), (("postln_alpha",), None, "postln_alpha"), (("logit_softcap",), -1.0, "softcap"),
                              (("layers", 0, "mixer", "q_temp", "every"), 0, "every"), (("layers", 1, "mixer", "q_rank"), None, "q_rank"),
                              (("layers",), [], "layers")]:
        bad = copy.deepcopy(CFG)
        node = bad
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        with pytest.raises(pe.ConfigError, match=word):
            pe.BurinexConfig.from_dict(bad)


def test_plan_names_every_tensor(pe):
    loader = import_module("pytorch-engine_b200.weights.loader")
    plan = pe.config.architecture("Burinex").plan(pe.BurinexConfig.from_dict(CFG))
    want, have = loader.expected_tensors(plan), plain.random_weights(CFG, 0)
    assert set(have) == set(want)
    for name, decl in want.items():
        assert decl.fits(have[name].shape), name
    assert plan.ignored == ("l1.norm2", "l1.ls2") and "ffn" not in plan.blocks[1].parts
    assert [b.arrangement for b in plan.blocks] == ["norm_of_sum"] * 4 and len(plan.positions) == 2
    assert plan.head.weights["weight"] == "head" and plan.head.params["softcap"] == 6.0


def test_cache_entries_are_keys_and_values_latent_rows_under_a_window_and_state(pe):
    plan = pe.config.architecture("Burinex").plan(pe.BurinexConfig.from_dict(CFG))
    reqs = {i: pe.parts.lookup("mixer", b.part("mixer").kind).cache_request(b.part("mixer").params) for i, b in enumerate(plan.blocks)}
    assert [r.kind for r in reqs.values()] == ["kv", "kv", "state", "kv"]
    assert (reqs[0].kv_heads, reqs[0].head_dim, reqs[0].value_dim) == (2, 10, 6)
    assert (reqs[1].head_dim, reqs[1].value_dim, reqs[1].window, reqs[1].values_in_keys) == (20, 14, 9, True)
    assert reqs[2].state_shapes == (("S", (2, 6, 8), "float32"),) and reqs[3].window is None
    cache = pe.cache.PagedCache(reqs, max_tokens=256, max_slots=2, max_seq_len=256, dtype=torch.float32, device="cpu")
    s = cache.alloc_slot()
    for n in (100, 130, 140):
        cache.reserve(s, n)
        cache.commit(s, n)
    held = {g.entries[0]: sum(p >= 0 for p in g.pages_of_slot[s]) for g in cache.groups if g.request.kind == "kv"}
    assert held == {0: 3, 1: 1, 3: 3}
    cache.free_slot(s)
    cache.check()


def test_exact_rotary_tables_with_scaled_frequencies(pe):
    class Rt:
        device = torch.device("cpu")
        position_limit = 5000
    sc = {"factor": 5.0, "original": 400, "fast": 12.0, "slow": 2.0}
    pos = pe.parts.lookup("position", "rope")({"rotary_dim": 20, "theta": 900.0, "max_positions": 10000, "style": "interleaved",
                                               "scaling": sc, "exact": True}, {}, Rt())
    cos, sin, dims = pos.tables()
    want = plain.rotary_tables({"dims": 20, "base": 900.0, "scaling": sc}, torch.arange(5000))
    assert dims == 20 and (cos - want[0]).abs().max() < 2e-7 and (sin - want[1]).abs().max() < 2e-7


def test_what_cannot_be_built_together_is_refused(pe):
    att = pe.parts.lookup("mixer", "attention")
    base = {"hidden": 8, "n_heads": 2, "n_kv_heads": 1, "head_dim": 4, "query_temperature": {"coef": 1.0, "every": 4}}
    w = {n: torch.zeros(s) for n, s in (("q_proj", (8, 8)), ("k_proj", (4, 8)), ("v_proj", (4, 8)), ("o_proj", (8, 8)), ("q_norm", (4,)),
                                        ("k_norm", (4,)), ("q_bias", (8,)), ("k_bias", (4,)), ("v_bias", (4,)))}
    rt = pe.parts.Runtime("cpu", torch.float32)
    for extra in ({"qk_norm": True}, {"bias": True}, {"qk_unit": True}, {"v_norm": "unit"}, {"query_temperature": {"coef": 1.0, "every": 0}}):
        with pytest.raises(ValueError):
            att(dict(base, **extra), w, rt)
    moe = pe.parts.lookup("feed_forward", "routed_experts")
    with pytest.raises(ValueError, match="identity"):
        moe({"hidden": 8, "n_experts": 0, "n_identity": 2, "top": 1, "intermediate": 4, "choice": "sigmoid_groups", "weight_on": "input"},
            {"router": torch.zeros(2, 8)}, rt)
    with pytest.raises(ValueError, match="decays"):
        pe.parts.lookup("mixer", "lightning")({"hidden": 8, "n_heads": 2, "head_dim": 4, "v_head_dim": 4, "decay": [0.5]}, {}, rt)


def _tokens(n, seed):
    return torch.randint(0, CFG["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def test_plain_implementation_is_causal_and_every_mechanism_matters():
    w = plain.random_weights(CFG, 5)
    toks = _tokens(40, 1)
    whole = plain.forward(CFG, w, toks)
    assert (whole[:25] - plain.forward(CFG, w, toks[:25])).abs().max() < 1e-9

    def differs(cfg, weights, least=1e-3):
        return (whole - plain.forward(cfg, weights, toks)).abs().max() > least

    for path, value in [(("layers", 0, "mixer", "q_temp", "coef"), 0.0), (("layers", 0, "mixer", "q_temp", "every"), 8),
                        (("layers", 1, "mixer", "mask", "size"), 8), (("layers", 1, "mixer", "mask", "size"), 10),
                        (("layers", 1, "mixer", "rot", "scaling", "factor"), 1.0), (("layers", 1, "mixer", "rot", "dims"), 4),
                        (("layers", 2, "mixer", "decay"), [0.6, 0.97]), (("layers", 0, "mlp", "router", "top"), 1),
                        (("layers", 0, "mlp", "shared"), None), (("postln_alpha",), 1.0), (("logit_softcap",), 12.0), (("norm", "eps"), 0.3),
                        (("layers", 3, "mixer", "scale"), 0.1)]:
        other = copy.deepcopy(CFG)
        node = other
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        assert differs(other, w), path
    for name in ("l0.ls1", "l0.ls2", "l0.mix.q.norm", "l0.mix.k.norm", "l0.mix.g", "l1.mix.dq.norm", "l1.mix.dkv.norm", "l1.mix.uk", "l1.mix.uv",
                 "l1.mix.sink", "l2.mix.norm", "l2.mix.g", "l2.mlp.router", "l0.mlp.shared.up", "l3.norm2", "final.norm"):
        other = dict(w)
        other[name] = w[name] * torch.linspace(0.2, 0.9, w[name].shape[0]).view([-1] + [1] * (w[name].dim() - 1))
        assert differs(CFG, other), name
    # rounding the products to bfloat16 moves the logits a little, not much
    with plain.stored(torch.bfloat16):
        rounded = plain.forward(CFG, w, toks)
    assert 1e-5 < float((whole - rounded).abs().median()) < 0.1 * float(whole.abs().max())


def test_the_plain_softmax_keeps_a_part_for_the_sink():
    seen = plain.visible_keys(4, None)
    assert torch.allclose(plain.sink_softmax(torch.zeros(4, 4), seen, 0.0).sum(1), torch.tensor([1 / 2, 2 / 3, 3 / 4, 4 / 5]))
    assert torch.allclose(plain.sink_softmax(torch.zeros(4, 4), seen, math.log(3.0)).sum(1), torch.tensor([1 / 4, 2 / 5, 3 / 6, 4 / 7]))
    assert plain.visible_keys(6, 3).sum(1).tolist() == [1, 2, 3, 3, 3, 3]


def test_the_temperature_steps_at_multiples():
    t = plain.temperature(torch.arange(9), {"coef": 2.0, "every": 4}, torch.float64)
    want = [1.0] * 3 + [1.0 + 2.0 * math.log(2.0)] * 4 + [1.0 + 2.0 * math.log(3.0)] * 2
    assert torch.allclose(t, torch.tensor(want, dtype=torch.float64))
