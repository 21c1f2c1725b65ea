"""What needs no GPU of the Bobasun architecture: its configuration file, its plan (tensor names, which layer keeps its values
and which mix them in), rotary tables with linearly scaled frequencies, and the plain implementation's own consistency."""
import copy
from importlib import import_module

import pytest
import torch

import plain_bobasun as plain

CFG = {"architecture": "Bobasun", "vocab": 71, "width": 36, "streams": 2, "norm": {"eps": 1e-4}, "embedding": {"scale": 1.5},
       "layers": [
           {"type": "attention", "mixer": {"heads": 2, "kv_heads": 1, "dim": 10, "vdim": 6, "scale": 0.4, "v_mix": False},
            "mlp": {"kind": "dense", "ff": 28, "limit": 1.0}},
           {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 8, "scale": 0.3, "v_mix": True,
                                           "rot": {"base": 500.0, "dims": 8, "scaling": {"factor": 3.0}}}, "mlp": None},
           {"type": "attention", "mixer": {"heads": 6, "kv_heads": 2, "dim": 8, "vdim": 8, "scale": 0.5, "v_mix": True,
                                           "rot": {"base": 90.0, "dims": 8}}, "mlp": {"kind": "dense", "ff": 20, "limit": 2.5}},
           {"type": "attention", "mixer": {"heads": 2, "kv_heads": 2, "dim": 16, "vdim": 8, "scale": 0.2, "v_mix": True,
                                           "rot": {"base": 500.0, "dims": 8, "scaling": {"factor": 3.0}}},
            "mlp": {"kind": "dense", "ff": 12, "limit": 0.7}}]}


def test_config_reads_every_layer_by_itself_and_writes_it_back(pe):
    cfg = pe.BobasunConfig.from_dict(CFG)
    assert (cfg.streams, cfg.embedding_scale, cfg.norm_eps, cfg.vocab_size) == (2, 1.5, 1e-4, 71)
    assert cfg.layers[0].mixer.rot_dims == 0 and not cfg.layers[0].mixer.v_mix and cfg.layers[1].mlp is None
    assert (cfg.layers[1].mixer.rot_factor, cfg.layers[2].mixer.rot_factor) == (3.0, 1.0)
    assert [layer.mlp.limit for layer in cfg.layers if layer.mlp] == [1.0, 2.5, 0.7]
    assert pe.BobasunConfig.from_dict(cfg.to_dict()) == cfg
    assert pe.config.architecture_of(CFG).name == "Bobasun"
    for path, value, word in [(("layers", 0, "type"), "delta", "type"), (("layers", 1, "mixer", "kv_heads"), 3, "multiple"),
                              (("layers", 1, "mixer", "rot", "dims"), 14, "dims"), (("layers", 1, "mixer", "rot", "dims"), 7, "even"),
                              (("layers", 0, "mlp", "kind"), "moe", "kind"), (("layers", 0, "mlp", "limit"), None, "limit"),
                              (("norm",), None, "norm"), (("streams",), 0, "streams"), (("layers", 2, "mixer", "v_mix"), 1, "v_mix"),
                              (("layers", 2, "mixer", "vdim"), 6, "v_mix"), (("layers",), [], "layers")]:
        bad = copy.deepcopy(CFG)
        node = bad
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        with pytest.raises(pe.ConfigError, match=word):
            pe.BobasunConfig.from_dict(bad)


def test_plan_names_every_tensor_and_the_first_mixing_layer_keeps_its_values(pe):
    loader = import_module("pytorch-engine_b200.weights.loader")
    plan = pe.config.architecture("Bobasun").plan(pe.BobasunConfig.from_dict(CFG))
    assert [b.part("mixer").params["value_mix"] for b in plan.blocks] == [None, "keep", "mix", "mix"]
    want = loader.expected_tensors(plan)
    have = plain.random_weights(CFG, 0)
    assert set(have) - set(want) == {"l1.mix.vmix"} and set(want) <= set(have)     # the first mixing layer's number is not used
    assert "l1.mix.vmix" in plan.ignored and "l0.mix.vmix" in plan.ignored and "l2.mix.vmix" not in plan.ignored
    assert "l1.norm2" in plan.ignored and "l1.hc2.mix" in plan.ignored
    for name, decl in want.items():
        assert decl.fits(have[name].shape), name
    assert [b.arrangement for b in plan.blocks] == ["streams"] * 4 and "ffn" not in plan.blocks[1].parts
    assert len(plan.positions) == 2 and plan.blocks[1].part("mixer").params["position"] == plan.blocks[3].part("mixer").params["position"]
    assert plan.head.weights["weight"] == "head" and plan.embedding.weights["weight"] == "embed"


def test_cache_entries_hold_keys_and_values_of_their_own_sizes(pe):
    plan = pe.config.architecture("Bobasun").plan(pe.BobasunConfig.from_dict(CFG))
    reqs = {i: pe.parts.lookup("mixer", "attention").cache_request(b.part("mixer").params) for i, b in enumerate(plan.blocks)}
    assert [(r.kv_heads, r.head_dim, r.value_dim) for r in reqs.values()] == [(1, 10, 6), (2, 12, 8), (2, 8, 8), (2, 16, 8)]
    cache = pe.cache.PagedCache(reqs, max_tokens=256, max_slots=2, max_seq_len=256, dtype=torch.float32, device="cpu")
    s = cache.alloc_slot()
    cache.reserve(s, 130)
    cache.commit(s, 130)
    assert all(len(g.pages_of_slot[s]) == 3 for g in cache.groups)
    cache.free_slot(s)
    cache.check()


def test_rotary_tables_with_linear_scaling(pe):
    class Rt:
        device = torch.device("cpu")
        position_limit = 300
    for exact in (True, False):
        pos = pe.parts.lookup("position", "rope")({"rotary_dim": 12, "theta": 700.0, "max_positions": 1000, "style": "neox",
                                                   "scaling": {"factor": 2.5}, "exact": exact}, {}, Rt())
        cos, sin, dims = pos.tables()
        assert dims == 12 and cos.shape == (300, 6)
        ang = torch.arange(300, dtype=torch.float64)[:, None] * (700.0 ** (-2.0 * torch.arange(6, dtype=torch.float64) / 12) / 2.5)
        tol = 1e-7 if exact else 2e-5
        assert (cos - torch.cos(ang)).abs().max() < tol and (sin - torch.sin(ang)).abs().max() < tol


def _tokens(n, seed):
    return torch.randint(0, CFG["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def test_plain_implementation_is_causal_and_every_mechanism_matters():
    w = plain.random_weights(CFG, 5)
    toks = _tokens(40, 1)
    whole = plain.forward(CFG, w, toks)
    assert (whole[:25] - plain.forward(CFG, w, toks[:25])).abs().max() < 1e-9

    def differs(cfg, weights, least=1e-3):
        return (whole - plain.forward(cfg, weights, toks)).abs().max() > least

    for path, value in [(("layers", 1, "mixer", "v_mix"), False), (("layers", 1, "mixer", "rot", "scaling", "factor"), 1.0),
                        (("layers", 2, "mlp", "limit"), 0.4), (("embedding", "scale"), 3.0), (("norm", "eps"), 0.3),
                        (("layers", 0, "mixer", "scale"), 0.1), (("layers", 3, "mixer", "rot", "dims"), 4)]:
        other = copy.deepcopy(CFG)
        node = other
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        assert differs(other, w), path
    for name in ("l0.mix.q.b", "l0.mix.k.b", "l0.mix.v.b", "l0.mix.o.b", "l0.mlp.gate.b", "l0.mlp.up.b", "l0.mlp.down.b", "l0.mix.g",
                 "l2.mix.vmix", "l3.hc1.in", "l3.hc1.out", "l3.hc2.mix", "l3.norm2"):
        other = dict(w)
        other[name] = w[name] * 0.5
        assert differs(CFG, other), name
    # the first mixing layer's own number is not used; the mix matrix is indexed [from, to]
    other = dict(w)
    other["l1.mix.vmix"] = w["l1.mix.vmix"] * 0.5
    assert not differs(CFG, other, 1e-12)
    other = dict(w)
    other["l0.hc1.mix"] = w["l0.hc1.mix"].T.contiguous()
    assert differs(CFG, other)
    # rounding the products to bfloat16 moves the logits a little, not much
    with plain.stored(torch.bfloat16):
        rounded = plain.forward(CFG, w, toks)
    assert 1e-5 < (whole - rounded).abs().max() < 0.2 * whole.abs().max()


def test_the_sink_of_the_plain_attention_keeps_a_part_of_the_weight():
    q, k, v = torch.zeros(4, 1, 2), torch.zeros(4, 1, 2), torch.ones(4, 1, 3)
    out = plain.sink_attention(q, k, v, 1.0)                       # all scores are 0: t + 1 keys beside the sink
    assert torch.allclose(out[:, 0, 0], torch.tensor([1 / 2, 2 / 3, 3 / 4, 4 / 5]))
    k[1] = 200.0
    q[3] = 1.0
    out = plain.sink_attention(q, k, v, 1.0)
    assert torch.allclose(out[3], torch.ones(1, 3))
    q[3] = -1.0                                                    # that one far below zero, the others at 0
    assert torch.allclose(plain.sink_attention(q, k, v, 1.0)[3], torch.full((1, 3), 3 / 4))


def test_random_model_weights_have_streams_near_the_identity(pe):
    rw = import_module("pytorch-engine_b200.weights.random_init")
    plan = pe.config.architecture("Bobasun").plan(pe.BobasunConfig.from_dict(CFG))
    w = rw.random_weights(plan, 3)
    assert (w["l0.hc1.mix"].float() - torch.eye(2)).abs().max() < 0.2
    assert 0.0 <= float(w["l0.hc1.in"].float().min()) and w["l2.mix.vmix"].shape == ()
