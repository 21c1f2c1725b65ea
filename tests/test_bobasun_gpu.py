"""The Bobasun architecture on the engine against the plain implementation in ``plain_bobasun.py``: mechanisms at kernel level
with inputs made so that a fault shows, every mechanism alone as a one-layer model, then whole models: prompts, token-by-token
decoding, prompts in portions, unequal batches, slots and pages used again, long decoding, generation through the entry point."""
import copy
import json

import pytest
import torch

import plain_bobasun as plain
from conftest import rel_err

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TOL = {"float32": 3e-5, "bfloat16": 2e-2}


def _att(heads, kv, dim, vdim, scale, dims=0, base=10000.0, factor=None, mix=False):
    d = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": mix}
    if dims:
        d["rot"] = {"base": base, "dims": dims}
        if factor:
            d["rot"]["scaling"] = {"factor": factor}
    return d


def _layer(mixer, ff=None, limit=1.0):
    return {"type": "attention", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


# The tests' own models.  A: nothing is a multiple of 8 anywhere (no kernel may take its 16-byte paths), five streams, value
# mixing from the second layer on, partial rotation with scaled frequencies, none, and whole, a layer without feed-forward.
# B: sizes that the tensor-core attention kernels take whole (64 and 128, the latter on tcgen05 in prompts), a feed-forward
# that the fused gate|up product takes, two streams, every layer mixes.  C: key and value sizes that run in padded tiles
# (below and above 64, 128 and 192), one stream, groups of 8 and 1, scale one.  D: small sizes in steps of 8, four streams, no
# mixing layer but one.  E: nine streams (the kernel without a fixed number of them).
CONFIGS = {
    "A": {"architecture": "Bobasun", "vocab": 131, "width": 54, "streams": 5, "norm": {"eps": 2e-5}, "embedding": {"scale": 3.0},
          "layers": [_layer(_att(3, 1, 14, 10, 0.4, 6, 100.0, 4.0), 37, 1.5), _layer(_att(4, 2, 10, 6, 0.5, mix=True)),
                     _layer(_att(2, 2, 18, 6, 0.3, 18, 3000.0, mix=True), 22, 0.6), _layer(_att(6, 2, 7, 6, 0.6, 4, 50.0, 1.7, mix=True), 31, 3.0)]},
    "B": {"architecture": "Bobasun", "vocab": 256, "width": 128, "streams": 2, "norm": {"eps": 1e-6}, "embedding": {"scale": 0.7},
          "layers": [_layer(_att(4, 2, 64, 64, 0.2, 64, 30000.0, 8.0, mix=True), 128, 1.0),
                     _layer(_att(8, 2, 128, 64, 0.15, 128, 10000.0, mix=True), 256, 2.5),
                     _layer(_att(4, 2, 128, 64, 0.1, 32, 500.0, 2.0, mix=True), 128, 0.5)]},
    "C": {"architecture": "Bobasun", "vocab": 90, "width": 64, "streams": 1, "norm": {"eps": 1e-5}, "embedding": {"scale": 5.0},
          "layers": [_layer(_att(8, 1, 72, 40, 0.2, 48, 1000.0, 3.0), 48), _layer(_att(2, 2, 120, 128, 0.12, 120, 20000.0), 96, 4.0),
                     _layer(_att(4, 1, 192, 56, 0.08, 64, 900.0, 16.0, mix=True)), _layer(_att(2, 1, 256, 56, 0.07, mix=True), 40, 0.8),
                     _layer(_att(3, 1, 32, 104, 1.0, 16, 100.0), 56, 1.2)]},
    "D": {"architecture": "Bobasun", "vocab": 77, "width": 48, "streams": 4, "norm": {"eps": 3e-6},
          "layers": [_layer(_att(2, 2, 24, 16, 0.4, 16, 5000.0), 40, 2.0), _layer(_att(4, 4, 8, 8, 0.5, 8, 60.0, 2.0, mix=True), 24, 1.0),
                     _layer(_att(5, 1, 40, 24, 0.3), 16, 0.9)]},
    "E": {"architecture": "Bobasun", "vocab": 60, "width": 40, "streams": 9, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0},
          "layers": [_layer(_att(2, 1, 16, 24, 0.4, 16, 100.0, 2.0, mix=True), 24), _layer(_att(2, 1, 16, 24, 0.4, 8, 100.0, mix=True), 32)]},
}
SEEDS = {"A": 31, "B": 32, "C": 33, "D": 34, "E": 35}


def _tokens(vocab, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


class Models:
    def __init__(self, pe):
        self.pe = pe
        self.configs = dict(CONFIGS)
        self.weights = {}
        self.engines = {}
        self.refs = {}

    def add(self, key, cfg, seed):
        self.configs[key] = cfg
        SEEDS[key] = seed

    def w(self, key):
        if key not in self.weights:
            self.weights[key] = plain.random_weights(self.configs[key], SEEDS[key])
        return self.weights[key]

    def engine(self, key, dtype, **kw):
        ident = (key, dtype, tuple(sorted(kw.items())))
        if ident not in self.engines:
            cfg = self.pe.BobasunConfig.from_dict(self.configs[key])
            args = dict(dtype=dtype, max_context_len=1024, max_cache_tokens=64 * 40, max_batch=8)
            args.update(kw)
            self.engines[ident] = self.pe.Engine(None, config=cfg, weights={k: v.to(DEV) for k, v in self.w(key).items()}, **args)
        return self.engines[ident]

    def ref(self, key, toks):
        ident = (key, tuple(toks))
        if ident not in self.refs:
            self.refs[ident] = plain.forward(self.configs[key], self.w(key), toks).float()
        return self.refs[ident]

    def noise(self, key, toks):
        """How far rounding to bfloat16 alone moves each position's logits (root mean square over the vocabulary)."""
        ident = (key, tuple(toks), "noise")
        if ident not in self.refs:
            with plain.stored(torch.bfloat16):
                rounded = plain.forward(self.configs[key], self.w(key), toks)
            self.refs[ident] = (rounded - self.ref(key, toks).double()).pow(2).mean(dim=1).sqrt()
        return self.refs[ident]

    def check(self, key, dtype, toks, got, positions, what):
        """float32: every logit within 3e-5 of the largest.  bfloat16: the error is held against what rounding alone does
        in the plain implementation: on average no more than twice that, and at no more than one position in fifty (or
        one) above three times the larger of that position's own figure and the average."""
        positions = list(positions)
        ref = self.ref(key, toks)[positions]
        got = got.float().cpu()
        assert got.shape == ref.shape, what
        if dtype == "float32":
            err = rel_err(got, ref)
            assert err < TOL[dtype], f"{what}: error {err:.3e} (limit {TOL[dtype]:.0e})"
            return
        noise = self.noise(key, toks)
        err = (got.double() - ref.double()).pow(2).mean(dim=1).sqrt()
        floor = float(noise.mean())
        limit = 2.0 * max(float(noise[positions].mean()), floor)
        assert float(err.mean()) <= limit, f"{what}: mean error {float(err.mean()):.3e}, limit {limit:.3e}"
        over = int((err > 3.0 * torch.clamp(noise[positions], min=floor)).sum())
        assert over <= max(1, len(positions) // 50), f"{what}: {over} of {len(positions)} positions beyond three times rounding"


@pytest.fixture(scope="module")
def models(pe):
    return Models(pe)


def _entry(pe, slot, toks, want):
    return pe.StepEntry(slot, toks, tuple(want))


# ---- mechanisms at kernel level -----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("s,width", [(1, 50), (2, 72), (3, 1028), (4, 200), (5, 64), (6, 33), (8, 48), (11, 60), (4, 5000)])
def test_streams_written_read_and_normed_in_one_pass(pe, dtype, s, width):
    """From one row that stands for all streams and from streams that exist, with and without a bias, each norm and none, all
    rows and chosen ones; the mix is neither symmetric nor near the identity, and the rows are far from zero mean."""
    ops = pe.kernels.ops
    g = torch.Generator().manual_seed(s * width)
    n = 19
    X = torch.randn(n, s, width, generator=g) * 2 + 3
    y = (torch.randn(n, width, generator=g) * 2).to(dtype)
    bias, w = torch.randn(width, generator=g), torch.randn(width, generator=g)
    mix, write, read = torch.randn(s, s, generator=g), torch.randn(s, generator=g), torch.randn(s, generator=g)
    rows = torch.tensor([5, 0, 18], dtype=torch.int32, device=DEV)
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    norms = {"layer": lambda u: plain.layer_norm(u, w.double(), 1e-5), "rms": lambda u: plain.unit(u, 1e-5) * w, None: lambda u: u}
    for from_one in (False, True):
        old = X[:, :1].expand(n, s, width).contiguous() if from_one else X
        for with_y in (True, False):
            for b in ((bias, None) if with_y else (None,)):
                new = old.double().transpose(0, 1)
                if with_y:
                    yy = y.double() + (0 if b is None else b.double())
                    new = plain.write_streams(new, yy, mix.double(), write.double())
                u = plain.read_streams(new, read.double())
                for norm, fn in norms.items():
                    for chosen in (None, rows):
                        x = torch.full_like(X, float("nan")).to(DEV) if from_one else X.clone().to(DEV)
                        before = x.clone()
                        out = torch.empty(n if chosen is None else 3, width, dtype=torch.float32 if norm is None else dtype, device=DEV)
                        ops.stream_mix(X[:, 0].contiguous().to(DEV) if from_one else None, x, y.to(DEV) if with_y else None,
                                       None if b is None else b.to(DEV), mix.to(DEV), write.to(DEV), read.to(DEV), norm,
                                       None if norm is None else w.to(DEV), 1e-5, out, chosen)
                        want = fn(u)[slice(None) if chosen is None else [5, 0, 18]]
                        err = (out.double().cpu() - want).abs().max() / want.abs().max()
                        assert err < (2e-5 if norm is None else tol), (from_one, with_y, norm, float(err))
                        if with_y and chosen is None:
                            assert (x.double().cpu() - new.transpose(0, 1)).abs().max() < 2e-5 * new.abs().max()
                        else:
                            assert torch.equal(x.nan_to_num(7.0), before.nan_to_num(7.0))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim", [50, 96])
def test_layer_norm_part_alone_and_behind_the_usual_add(pe, dtype, dim):
    g = torch.Generator().manual_seed(dim)
    rt = pe.parts.Runtime(torch.device(DEV), dtype)
    w = torch.randn(dim, generator=g)
    part = pe.parts.lookup("norm", "layer_norm")({"dim": dim, "eps": 0.02}, {"weight": w.to(DEV)}, rt)
    x, d = torch.randn(23, dim, generator=g) * 0.2 + 5, (torch.randn(23, dim, generator=g)).to(dtype)
    tol = 1e-4 if dtype == torch.float32 else 4e-2
    stream, out = x.clone().to(DEV), torch.empty(23, dim, dtype=dtype, device=DEV)
    part.add_forward(stream, d.to(DEV), out)
    want = plain.layer_norm(x.double() + d.double(), w.double(), 0.02)
    assert (stream.cpu() - (x + d.float())).abs().max() < 1e-5 and (out.double().cpu() - want).abs().max() < tol
    rows = torch.tensor([22, 3], dtype=torch.int32, device=DEV)
    few = torch.empty(2, dim, dtype=dtype, device=DEV)
    part.add_forward(stream, None, few, rows)
    assert (few.double().cpu() - want[[22, 3]]).abs().max() < tol
    xd = x.to(dtype)
    assert (part.forward(xd.to(DEV)).double().cpu() - plain.layer_norm(xd.double(), w.double(), 0.02)).abs().max() < tol


class Pages:
    """A hand-made paged cache for kernel tests: sequence b's logical page i is physical page ``table[b][i]``."""

    def __init__(self, lens, kvh, d, dv, seed=0, fill=0.0):
        g = torch.Generator().manual_seed(seed)
        n_pages = sum(-(-n // 64) for n in lens) + 3
        order = torch.randperm(n_pages, generator=g).tolist()
        self.table = torch.full((len(lens), max(-(-n // 64) for n in lens) + 1), -1, dtype=torch.int32)
        for b, n in enumerate(lens):
            for i in range(-(-n // 64)):
                self.table[b, i] = order.pop()
        self.k = torch.full((n_pages, kvh, 64, d), fill)
        self.v = torch.full((n_pages, kvh, 64, dv), fill)
        self.n_pages = n_pages

    def put(self, b, k, v):
        """``k [n, kvh, d]``, ``v [n, kvh, dv]`` at positions 0 .. n - 1."""
        for pos in range(k.shape[0]):
            page = int(self.table[b, pos // 64])
            self.k[page, :, pos % 64] = k[pos]
            self.v[page, :, pos % 64] = v[pos]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,d,dv,rot", [(3, 1, 14, 10, 6), (4, 2, 64, 64, 64), (6, 2, 72, 40, 32), (2, 1, 256, 128, 0), (5, 5, 24, 8, 16),
                                             (8, 2, 128, 64, 128), (2, 2, 40, 24, 24)])
def test_bias_rotation_unit_norm_mixed_values_and_the_append(pe, dtype, nh, nkv, d, dv, rot):
    """Two sequences of unequal length that go on from unequal positions, few tokens and many; the first pass keeps its values,
    the second mixes them in.  Queries come back in place, keys and values must lie in their pages, nothing else may change
    but the rest of a sequence's last page, which is cleared."""
    ops = pe.kernels.ops
    g = torch.Generator().manual_seed(nh * d + dv)
    rt = pe.parts.Runtime(torch.device(DEV), dtype)
    factor = 2.5
    m = {"rot": {"base": 300.0, "dims": rot, "scaling": {"factor": factor}}} if rot else {}
    cos = sin = None
    if rot:
        cos, sin, _ = pe.parts.lookup("position", "rope")({"rotary_dim": rot, "theta": 300.0, "max_positions": 700, "style": "neox",
                                                           "scaling": {"factor": factor}, "exact": True}, {}, rt).tables()
    for lens, pasts in (([5, 9], [60, 0]), ([1, 1], [64, 127]), ([290, 70], [3, 65])):
        n = sum(lens)
        width = (nh + nkv) * d + nkv * dv + 8
        ld = -(-width // 8) * 8
        proj = torch.randn(n, ld, generator=g).to(dtype)
        bias = torch.randn((nh + nkv) * d + nkv * dv, generator=g)
        pages = Pages([p + q for p, q in zip(pasts, lens)], nkv, d, dv, seed=d, fill=7.0)
        kp, vp = pages.k.to(DEV, dtype), pages.v.to(DEV, dtype)
        qstart = torch.tensor([0, lens[0], n], dtype=torch.int32, device=DEV)
        seq = torch.tensor([0] * lens[0] + [1] * lens[1], dtype=torch.int32, device=DEV)
        pos = torch.tensor([p + i for p, q in zip(pasts, lens) for i in range(q)], dtype=torch.int32, device=DEV)
        slots = torch.tensor([0, 1], dtype=torch.int32, device=DEV)
        status = torch.zeros(4, dtype=torch.int32, device=DEV)
        kept = torch.full((n, nkv * dv), float("nan"), dtype=dtype, device=DEV)
        first = (torch.randn(n, nkv * dv, generator=g)).to(dtype)
        for mode in ("keep", "mix"):
            qkv = proj.clone().to(DEV)
            ops.qkv_rotate_append(qkv, n, nh, nkv, d, dv, None, None, 0.01, cos, sin, rot, False, False, None, None, 0, False, seq, pos,
                                  slots, qstart, pages.table.to(DEV), pages.n_pages, kp, vp, True, status, bias.to(DEV), qk_unit=True,
                                  v_mix=first.to(DEV) if mode == "mix" else None, v_lambda=0.3, v_keep=kept if mode == "keep" else None)
            x = proj[:, :bias.numel()].double() + bias.double()
            cpos = pos.cpu()
            q = plain.unit(plain.rotate(x[:, :nh * d].view(n, nh, d), cpos, m.get("rot")), 0.01)
            k = plain.unit(plain.rotate(x[:, nh * d:(nh + nkv) * d].view(n, nkv, d), cpos, m.get("rot")), 0.01)
            v = x[:, (nh + nkv) * d:].view(n, nkv, dv)
            if mode == "mix":
                v = plain.mix_values(v, first.double().view(n, nkv, dv), 0.3)
            tol = 2e-5 if dtype == torch.float32 else 2e-2
            assert (qkv[:, :nh * d].double().cpu().view(n, nh, d) - q).abs().max() < tol * float(q.abs().max())
            assert torch.equal(qkv[:, bias.numel():].cpu(), proj[:, bias.numel():])
            if mode == "keep":
                assert (kept.double().cpu().view(n, nkv, dv) - v).abs().max() < tol * float(v.abs().max())
            kc, vc = kp.double().cpu(), vp.double().cpu()
            t = 0
            for b in range(2):
                for i in range(lens[b]):
                    p = pasts[b] + i
                    page = int(pages.table[b, p // 64])
                    assert (kc[page, :, p % 64] - k[t]).abs().max() < tol * float(k.abs().max()), (mode, b, i)
                    assert (vc[page, :, p % 64] - v[t]).abs().max() < tol * float(v.abs().max()), (mode, b, i)
                    t += 1
                last = pasts[b] + lens[b] - 1
                page = int(pages.table[b, last // 64])
                if lens[b] > 1 or last % 64 == 0:
                    assert float(kc[page, :, last % 64 + 1:].abs().sum()) == 0.0 and float(vc[page, :, last % 64 + 1:].abs().sum()) == 0.0
                for p in range(pasts[b] // 64 * 64, pasts[b]):       # what was there before stays
                    assert float(kc[int(pages.table[b, p // 64]), :, p % 64].min()) == 7.0
        assert status.tolist()[0] == 0


@pytest.mark.parametrize("nh,nkv,extra,rot", [(4, 2, 8, 128), (3, 1, 0, 0), (6, 3, 16, 128), (2, 2, 264, 128)])
def test_the_products_epilogue_does_what_the_separate_kernel_does(pe, nh, nkv, extra, rot):
    """q|k|v|extra product with biases, rotation, unit norm, kept or mixed values and the append in its epilogue, against the
    plain equations and (for every page and every column) the separate kernel behind the same product."""
    ops = pe.kernels.ops
    bf, d, K = torch.bfloat16, 128, 192
    g = torch.Generator().manual_seed(nh + extra)
    rt = pe.parts.Runtime(torch.device(DEV), bf)
    cos = sin = None
    if rot:
        cos, sin, _ = pe.parts.lookup("position", "rope")({"rotary_dim": rot, "theta": 300.0, "max_positions": 900, "style": "neox",
                                                           "scaling": {"factor": 2.5}, "exact": True}, {}, rt).tables()
    lens, pasts = [300, 1, 70], [3, 64, 65]
    n, feats = sum(lens), (nh + 2 * nkv) * d
    x = torch.randn(n, K, generator=g).to(bf).to(DEV)
    w = (torch.randn(feats + extra, K, generator=g) * 0.2).to(bf).to(DEV)
    bias = torch.randn(feats, generator=g).to(DEV)
    first = torch.randn(n, nkv * d, generator=g).to(bf).to(DEV)
    qstart = torch.tensor([0, 300, 301, n], dtype=torch.int32, device=DEV)
    seq = torch.tensor([b for b in range(3) for _ in range(lens[b])], dtype=torch.int32, device=DEV)
    pos = torch.tensor([p + i for p, q in zip(pasts, lens) for i in range(q)], dtype=torch.int32, device=DEV)
    slots = torch.arange(3, dtype=torch.int32, device=DEV)
    status = torch.zeros(4, dtype=torch.int32, device=DEV)
    for mode in ("keep", "mix"):
        results = []
        for fused in (True, False):
            pages = Pages([p + q for p, q in zip(pasts, lens)], nkv, d, d, seed=1, fill=7.0)
            kp, vp = pages.k.to(DEV, bf), pages.v.to(DEV, bf)
            qkv = torch.zeros(n, feats + extra, dtype=bf, device=DEV)
            kept = torch.zeros(n, nkv * d, dtype=bf, device=DEV)
            where = (seq, pos, slots, qstart, pages.table.to(DEV), pages.n_pages, kp, vp)
            more = dict(qk_unit=True, v_mix=first if mode == "mix" else None, v_lambda=0.3, v_keep=kept if mode == "keep" else None)
            if fused:
                ops.gemm_umma2_qkv_rope(x, w, qkv, nh, nkv, d, None, None, 0.01, cos, sin, rot, *where, True, status, bias, **more)
            else:
                ops.gemm_umma2(x, w, qkv, status)
                ops.qkv_rotate_append(qkv, n, nh, nkv, d, d, None, None, 0.01, cos, sin, rot, False, False, None, None, 0, False, *where, True,
                                      status, bias, **more)
            results.append([t.float().cpu() for t in (qkv[:, :nh * d], qkv[:, feats:], kp, vp, kept)])
        for a, b in zip(*results):
            assert (a - b).abs().max() <= 2e-2 * max(float(b.abs().max()), 1e-3) if b.numel() else True
        y = (x.double() @ w.double().T).cpu()
        q = plain.unit(plain.rotate((y[:, :nh * d] + bias[:nh * d].double().cpu()).view(n, nh, d), pos.cpu(),
                                    {"base": 300.0, "dims": rot, "scaling": {"factor": 2.5}} if rot else None), 0.01)
        assert (results[0][0].double().view(n, nh, d) - q).abs().max() < 2e-2 * float(q.abs().max())
    assert status.tolist()[0] == 0


ATT_KERNELS = {"float32 arithmetic": [(3, 1, 14, 10), (6, 2, 72, 40)],
               "mma": [(4, 2, 64, 64), (8, 2, 128, 128), (6, 2, 72, 40), (4, 1, 8, 8), (3, 3, 24, 128), (5, 1, 136, 64), (16, 1, 192, 120),
                       (2, 2, 256, 16), (4, 4, 104, 72), (2, 1, 200, 128)],
               "umma": [(8, 2, 128, 128), (4, 2, 192, 128), (7, 1, 136, 40), (2, 2, 256, 128), (6, 3, 200, 8), (4, 1, 72, 40), (6, 2, 120, 128), (5, 5, 128, 64), (20, 1, 104, 72), (3, 1, 80, 8)]}


@pytest.mark.parametrize("kernel,nh,nkv,d,dv", [(k, *s) for k, shapes in ATT_KERNELS.items() for s in shapes])
@pytest.mark.parametrize("decode", [False, True])
def test_attention_with_a_sink_and_gates_sees_every_key_and_no_more(pe, decode, kernel, nh, nkv, d, dv):
    """One key matches the last query far better than the rest, at places before, on and behind page borders and at the first
    and the last position: the output is that key's value times the head's gate.  With the match one position behind the
    query the output must be the plain average of what is visible.  Keys that all score far below zero leave the weight to
    the sink: the output is nearly zero.  Then random keys."""
    if kernel == "umma" and decode:
        pytest.skip("a kernel for prompts")
    ops = pe.kernels.ops
    dt = torch.float32 if kernel == "float32 arithmetic" else torch.bfloat16
    g = torch.Generator().manual_seed(d + dv)
    status = torch.zeros(4, dtype=torch.int32, device=DEV)

    def run(lens, q_lens, q, ks, vs, scale):
        """``q`` rows of all the step's tokens, ``ks[b] [len, nkv, d]``: outputs of the kernel."""
        pages = Pages(lens, nkv, d, dv, seed=lens[0])
        for b, (k, v) in enumerate(zip(ks, vs)):
            pages.put(b, k, v)
        n = sum(q_lens)
        row = -(-(nh * d + nh) // 8) * 8
        rows = torch.zeros(n, row)
        rows[:, :nh * d] = q.reshape(n, nh * d)
        gate = torch.randn(n, nh, generator=g)
        rows[:, nh * d:nh * d + nh] = gate
        rows = rows.to(DEV, dt)
        qstart = torch.tensor([0] + torch.tensor(q_lens).cumsum(0).tolist(), dtype=torch.int32, device=DEV)
        past = torch.tensor([a - b for a, b in zip(lens, q_lens)], dtype=torch.int32, device=DEV)
        slots = torch.arange(len(lens), dtype=torch.int32, device=DEV)
        where = (qstart, past, slots, pages.table.to(DEV), pages.n_pages, pages.k.to(DEV, dt), pages.v.to(DEV, dt))
        out = torch.full((n, nh * dv), float("nan"), dtype=dt, device=DEV)
        gcol = rows[:, nh * d:nh * d + nh]
        splits = max(-(-x // 64) for x in lens)
        scratch = torch.full((ops.attention_generic_scratch_floats(len(lens), nh, dv, max(splits, 3)),), float("nan"), device=DEV)
        if kernel == "umma":
            ops.attention_umma_prefill(rows, out, len(lens), max(q_lens), nh, nkv, d, scale, 0, *where, status, sink=True, v_dim=dv, gate=gcol)
        elif kernel == "mma":
            ops.attention_mma_gated(decode, rows, out, len(lens), max(q_lens), nh, nkv, d, dv, scale, 0, *where, scratch, 64, splits, status,
                                    sink=True, gate=gcol)
            if decode:                                     # three even ranges give the same
                again = torch.full_like(out, float("nan"))
                ops.attention_mma_gated(decode, rows, again, len(lens), max(q_lens), nh, nkv, d, dv, scale, 0, *where, scratch, 0, 3, status,
                                        sink=True, gate=gcol)
                assert (again.float() - out.float()).abs().max() < 2e-2
        else:
            raw = torch.empty_like(out)
            ops.attention_generic_ex(decode, rows, raw, len(lens), max(q_lens), nh, nkv, d, dv, scale, 0, True, None, None, 0, False, *where,
                                     scratch, 64, splits, status)
            ops.sigmoid_gate(raw.view(n, nh, dv).transpose(0, 1), gcol, out)
        return out.double().cpu().view(n, nh, dv), torch.sigmoid(gcol.double().cpu())[:, :, None]

    tol = 1e-4 if dt == torch.float32 else 3e-2
    for n in (1, 64, 65, 300):
        i = n - 1
        nq = 1 if decode else min(5, n)
        for target in sorted({0, 63, 64, n // 2, i - 1, i, n}):
            if target < 0:
                continue
            k = torch.zeros(n, nkv, d)
            vals = torch.randn(n, nkv, dv, generator=g)
            if target < n:
                k[target, :, 0] = 1.0
                if target < n - 1:
                    k[target, :, d - 1] = -1.0            # (the last feature counts too)
            q = torch.zeros(nq, nh, d)
            q[:, :, 0] = 30.0
            q[:, :, d - 1] = -30.0 if target < n - 1 else 0.0
            out, gate = run([n], [nq], q, [k], [vals], 1.0)
            want = vals[target] if target < n else vals.sum(0) / (n + 1)
            want = want.repeat_interleave(nh // nkv, dim=0).double() * gate[-1]
            assert (out[-1] - want).abs().max() < tol, (n, target)
        k = torch.full((n, nkv, d), -1.0)
        out, _ = run([n], [nq], torch.full((nq, nh, d), 20.0 / d), [k], [torch.randn(n, nkv, dv, generator=g)], 1.0)
        assert out.abs().max() < 1e-5
    # random keys, three sequences of unequal length in one step
    lens = [200, 1, 77]
    q_lens = [1, 1, 1] if decode else [130, 1, 40]
    ks = [torch.randn(x, nkv, d, generator=g).to(dt).float() for x in lens]
    vs = [torch.randn(x, nkv, dv, generator=g).to(dt).float() for x in lens]
    q = torch.randn(sum(q_lens), nh, d, generator=g).to(dt).float()
    out, gate = run(lens, q_lens, q, ks, vs, d ** -0.5)
    at = 0
    for x, ql, k, v in zip(lens, q_lens, ks, vs):
        full = torch.zeros(x, nh, d, dtype=torch.float64)
        full[x - ql:] = q[at:at + ql].double()
        want = plain.sink_attention(full, k.double(), v.double(), d ** -0.5)[x - ql:] * gate[at:at + ql]
        assert (out[at:at + ql] - want).abs().max() < (1e-5 if dt == torch.float32 else 2e-2), (x, ql)
        at += ql
    assert status.tolist()[0] == 0


def test_clamped_gate_with_biases_in_every_product(pe):
    """Sums far beyond the limit on both sides (the gate only from above), per product kernel; unaligned and ragged sizes in
    the separate kernel."""
    ops = pe.kernels.ops
    g = torch.Generator().manual_seed(3)
    status = torch.zeros(4, dtype=torch.int32, device=DEV)
    for m, k, n, kernels in ((1, 96, 40, "s"), (8, 200, 128, "s"), (13, 64, 256, "su"), (130, 128, 128, "up"), (300, 192, 384, "up")):
        x = torch.randn(m, k, generator=g).to(torch.bfloat16)
        w = (torch.randn(2 * n, k, generator=g) * 0.3).to(torch.bfloat16)
        bias = torch.randn(2 * n, generator=g)
        y = x.double() @ w.double().T + bias.double()
        assert float(y[:, :n].max()) > 1.3 and float(y[:, n:].min()) < -1.3
        want = plain.clamped_glu(y[:, :n], y[:, n:], 1.3)
        for kind in kernels:
            out = torch.full((m, n), float("nan"), dtype=torch.bfloat16, device=DEV)
            glu = ("clamped_swish", 1.3, plain.SWISH_SLOPE, bias.to(DEV))
            if kind == "s":
                ops.gemm_smallm(x.to(DEV), w.to(DEV), out, pair_offset=n, glu=glu)
            else:
                (ops.gemm_umma if kind == "u" else ops.gemm_umma2)(x.to(DEV), w.to(DEV), out, status, pair_offset=n, glu=glu)
            assert (out.double().cpu() - want).abs().max() < 2e-2, (m, k, n, kind)
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        for n in (40, 37):
            gu = (torch.randn(21, 2 * n, generator=g) * 3).to(dtype)
            bias = torch.randn(2 * n, generator=g)
            out = torch.empty(21, n, dtype=dtype, device=DEV)
            for b in (bias, None):
                ops.glu_act(gu.to(DEV), out, "clamped_swish", 0.8, plain.SWISH_SLOPE, None if b is None else b.to(DEV))
                y = gu.double() + (0 if b is None else b.double())
                assert (out.double().cpu() - plain.clamped_glu(y[:, :n], y[:, n:], 0.8)).abs().max() < tol
    assert status.tolist()[0] == 0


def test_a_far_key_among_hundreds_through_rotation_and_unit_norm(pe, models):
    """A one-layer model made so that position 3 stands out for the last query of a 500-token prompt (the features that carry
    the match lie behind ``rot.dims``): nearly all weight on one far key, in a prompt and when the last token is decoded."""
    key = "far key"
    cfg = {"architecture": "Bobasun", "vocab": 64, "width": 32, "streams": 2, "norm": {"eps": 1e-5},
           "layers": [_layer(_att(2, 1, 16, 16, 1.0, 8, 100.0))]}
    models.add(key, cfg, 77)
    w = models.w(key)
    # token 7 appears at position 3 only and token 5 as the last token only; the key projection copies feature 0 (large for
    # token 7) and the query projection feature 1 (large for token 5) into one unrotated head feature.  All other keys and
    # queries are one and the same bias vector in other features, so that their unit vectors are at right angles to the match.
    w["embed"][:] = w["embed"] * 0.05
    w["embed"][7, 0] = w["embed"][5, 1] = 4.0
    for n in ("q", "k"):
        w[f"l0.mix.{n}"].zero_()
        w[f"l0.mix.{n}.b"].zero_()
    w["l0.norm1"].fill_(1.0)
    w["l0.mix.q.b"][13] = w["l0.mix.q.b"][29] = 0.5
    w["l0.mix.k.b"][14] = 0.5
    w["l0.mix.q"][12, 1] = w["l0.mix.q"][28, 1] = 8.0
    w["l0.mix.k"][12, 0] = 8.0
    w["l0.mix.v"] *= 10.0
    toks = [t if t not in (5, 7) else 8 for t in _tokens(64, 500, 5)]
    toks[3], toks[-1] = 7, 5
    for dtype in ("float32", "bfloat16"):
        eng = models.engine(key, dtype)
        s = eng.alloc_slot()
        whole = eng.step([_entry(pe, s, toks, [499])]).clone()
        eng.free_slot(s)
        s = eng.alloc_slot()
        eng.step([_entry(pe, s, toks[:499], [])])
        alone = eng.step([_entry(pe, s, toks[499:], [0])]).clone()
        eng.free_slot(s)
        models.check(key, dtype, toks, whole, [499], "far key in a prompt")
        models.check(key, dtype, toks, alone, [499], "far key decoded")
    # the case the test is for: without position 3 the logits differ
    other = list(toks)
    other[3] = 9
    assert rel_err(plain.forward(cfg, w, other)[499:].float(), models.ref(key, toks)[499:]) > 1e-2


# ---- every mechanism alone, as a model of one or two layers -----------------------------------------------------------
_TINY = _att(1, 1, 8, 8, 0.5)
ALONE = {
    "rotation scaled": [_layer(_att(4, 1, 24, 16, 0.5, 12, 500.0, 4.0))],
    "rotation whole": [_layer(_att(2, 2, 16, 40, 0.25, 16, 100.0))],
    "no rotation": [_layer(_att(2, 1, 12, 20, 0.4))],
    "tcgen05 sizes": [_layer(_att(8, 2, 128, 128, 0.09, 64, 10000.0, 16.0))],
    "tcgen05 padded": [_layer(_att(4, 2, 88, 32, 0.12, 88, 10000.0, 3.0))],
    "values mixed": [_layer(_att(2, 1, 8, 24, 0.5, mix=True)), _layer(_att(4, 1, 16, 24, 0.5, mix=True)), _layer(_att(3, 1, 8, 24, 0.5, mix=True))],
    "values mixed past a layer without": [_layer(_att(2, 2, 8, 6, 0.5, mix=True)), _layer(_att(4, 1, 16, 10, 0.5)),
                                          _layer(_att(2, 2, 8, 6, 0.5, mix=True))],
    "feed-forward": [_layer(_TINY, 40, 0.4)],
    "feed-forward wide": [_layer(_TINY, 256, 1.1)],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_one_mechanism_alone_whole_and_token_by_token(pe, models, name, dtype):
    key = "alone " + name
    cfg = {"architecture": "Bobasun", "vocab": 90, "width": 64, "streams": 2, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0},
           "layers": copy.deepcopy(ALONE[name])}
    models.add(key, cfg, 40 + sorted(ALONE).index(name))
    eng = models.engine(key, dtype, max_cache_tokens=64 * 12)
    toks = _tokens(90, 150, 9)
    s = eng.alloc_slot()
    got = eng.step([_entry(pe, s, toks, range(150))]).clone()
    eng.free_slot(s)
    models.check(key, dtype, toks, got, range(150), f"{name} whole")
    s = eng.alloc_slot()
    rows = [eng.step([_entry(pe, s, toks[:3], [2])]).clone()]
    for t in toks[3:150]:
        rows.append(eng.step([_entry(pe, s, [t], [0])]).clone())
    eng.free_slot(s)
    models.check(key, dtype, toks, torch.cat(rows), range(2, 150), f"{name} token by token")


def test_streams_blocks_beside_blocks_of_another_arrangement(pe):
    """A streams block, a pre-norm block with the usual single stream (it reads the sum), then streams again, under a norm the
    streams kernel knows (RMS) and one it does not (Dynamic Tanh); against the same order written out."""
    parts = pe.parts
    spec = parts.spec
    W, V = 24, 40
    g = torch.Generator().manual_seed(2)
    w = {}

    def put(name, *shape, s=1.0, base=0.0):
        w[name] = (base + s * torch.randn(shape, generator=g)).to(torch.bfloat16).float()
        return name

    def norm(kind, name):
        if kind == "dynamic_tanh":
            return spec.PartSpec(kind, {"dim": W}, {"weight": put(name, W, s=0.2, base=1.0), "bias": put(name + ".b", W, s=0.1),
                                                    "alpha": put(name + ".a", s=0.0, base=0.5)})
        return spec.PartSpec(kind, {"dim": W, "eps": 1e-5}, {"weight": put(name, W, s=0.2, base=1.0)})

    def ff(name):
        names = {"gate_proj": put(name + ".g", 32, W, s=0.3), "up_proj": put(name + ".u", 32, W, s=0.3), "down_proj": put(name + ".d", W, 32, s=0.3),
                 "gate_bias": put(name + ".gb", 32), "up_bias": put(name + ".ub", 32), "down_bias": put(name + ".db", W)}
        return spec.PartSpec("swiglu", {"hidden": W, "intermediate": 32, "activation": "clamped_swish", "limit": 1.0,
                                        "alpha": plain.SWISH_SLOPE, "bias": True}, names)

    def mixer(name):
        names = {f"{p}_proj": put(f"{name}.{p}", r, c, s=0.3) for p, r, c in (("q", 16, W), ("k", 8, W), ("v", 8, W), ("o", W, 16), ("g", 2, W))}
        names.update({f"{p}_bias": put(f"{name}.{p}b", r) for p, r in (("q", 16), ("k", 8), ("v", 8), ("o", W))})
        return spec.PartSpec("attention", {"hidden": W, "n_heads": 2, "n_kv_heads": 1, "head_dim": 8, "qk_norm": False, "qk_unit": True,
                                           "eps": 1e-5, "scale": 0.5, "position": None, "sink": True, "bias": True, "out_bias": True,
                                           "output_gate": "sigmoid_head"}, names)

    def bundle(name, s):
        return spec.PartSpec("stream_bundle", {"streams": s}, {"read": put(name + ".r", s), "mix": put(name + ".m", s, s, s=0.5),
                                                               "write": put(name + ".w", s)})

    kinds = [("layer_norm", 3), ("rmsnorm", 0), ("rmsnorm", 3), ("dynamic_tanh", 2)]
    blocks = []
    for i, (kind, s) in enumerate(kinds):
        p = {"mixer_norm": ("norm", norm(kind, f"{i}.n1")), "mixer": ("mixer", mixer(f"{i}.mix")), "ffn_norm": ("norm", norm(kind, f"{i}.n2")),
             "ffn": ("feed_forward", ff(f"{i}.ff"))}
        if s:
            p["mixer_streams"], p["ffn_streams"] = ("stream", bundle(f"{i}.h1", s)), ("stream", bundle(f"{i}.h2", s))
        blocks.append(spec.BlockSpec("streams" if s else "pre_norm", p))
    plan = spec.ModelPlan(hidden_size=W, vocab_size=V, max_positions=256,
                          embedding=spec.PartSpec("token_embedding", {"vocab": V, "hidden": W}, {"weight": put("e", V, W)}),
                          blocks=tuple(blocks), order=tuple(spec.RunStep(i) for i in range(4)), final_norm=norm("rmsnorm", "fn"),
                          head=spec.PartSpec("linear_head", {"vocab": V, "hidden": W}, {"weight": put("h", V, W)}))
    rt = parts.Runtime(torch.device(DEV), torch.float32)
    from importlib import import_module
    model = import_module("pytorch-engine_b200.engine.model").DecoderModel(plan, {k: v.to(DEV) for k, v in w.items()}, rt)
    runner = import_module("pytorch-engine_b200.engine.runner").ModelRunner
    cache = pe.cache.PagedCache(model.cache_requests(), max_tokens=512, max_slots=2, max_seq_len=256, dtype=torch.float32, device=DEV)
    run = runner(model, cache)
    toks = _tokens(V, 70, 3)
    s = run.alloc_slot()
    got = [run.step([_entry(pe, s, toks[:40], range(40))]).clone()]
    for t in toks[40:]:
        got.append(run.step([_entry(pe, s, [t], [0])]).clone())
    d = {k: v.double() for k, v in w.items()}

    def normed(kind, name, x):
        if kind == "layer_norm":
            return plain.layer_norm(x, d[name], 1e-5)
        if kind == "rmsnorm":
            return plain.unit(x, 1e-5) * d[name]
        return torch.tanh(d[name + ".a"] * x) * d[name] + d[name + ".b"]

    def attend(h, p):
        n = h.shape[0]
        q, k, v = (h @ d[f"{p}.{c}"].T + d[f"{p}.{c}b"] for c in "qkv")
        o = plain.sink_attention(plain.unit(q.view(n, 2, 8), 1e-5), plain.unit(k.view(n, 1, 8), 1e-5), v.view(n, 1, 8), 0.5)
        o = o * torch.sigmoid(h @ d[f"{p}.g"].T)[:, :, None]
        return o.reshape(n, 16) @ d[f"{p}.o"].T + d[f"{p}.ob"]

    def feed(h, p):
        return plain.clamped_glu(h @ d[f"{p}.g"].T + d[f"{p}.gb"], h @ d[f"{p}.u"].T + d[f"{p}.ub"], 1.0) @ d[f"{p}.d"].T + d[f"{p}.db"]

    x = d["e"][torch.tensor(toks)]
    X = None
    for i, (kind, n_streams) in enumerate(kinds):
        subs = [(f"{i}.n1", f"{i}.h1", lambda h: attend(h, f"{i}.mix")), (f"{i}.n2", f"{i}.h2", lambda h: feed(h, f"{i}.ff"))]
        if X is not None and X.shape[0] != n_streams:      # another number of streams, or one: they are summed
            x, X = X.sum(0), None
        for nm, hc, sub in subs:
            if n_streams == 0:
                x = x + sub(normed(kind, nm, x))
            else:
                X = torch.stack([x] * n_streams) if X is None else X
                X = plain.write_streams(X, sub(normed(kind, nm, plain.read_streams(X, d[hc + ".r"]))), d[hc + ".m"], d[hc + ".w"])
    want = normed("rmsnorm", "fn", X.sum(0)) @ d["h"].T
    assert rel_err(torch.cat(got).cpu(), want.float()) < 3e-5


# ---- whole models -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", sorted(CONFIGS))
def test_whole_prompt_and_its_first_tokens(pe, models, key, dtype):
    eng = models.engine(key, dtype)
    toks = _tokens(CONFIGS[key]["vocab"], 300, 1)
    ref = models.ref(key, toks)
    s = eng.alloc_slot()
    got = eng.step([_entry(pe, s, toks, range(300))]).clone()
    eng.free_slot(s)
    models.check(key, dtype, toks, got, range(300), f"{key} whole prompt")
    s = eng.alloc_slot()                               # a prompt of one token, on the slot that was just freed
    one = eng.step([_entry(pe, s, toks[:1], [0])]).clone()
    eng.free_slot(s)
    err = rel_err(one.cpu(), ref[:1])
    assert err < TOL[dtype], f"{key} one token on a used slot: {err:.3e}"
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", sorted(CONFIGS))
def test_long_token_by_token_decoding_equals_the_prompt(pe, models, key, dtype):
    """A short prompt, then 240 tokens one by one (over three page borders, through CUDA graphs), against the plain
    implementation of the whole sequence."""
    eng = models.engine(key, dtype)
    toks = _tokens(CONFIGS[key]["vocab"], 255, 2)
    s = eng.alloc_slot()
    rows = [eng.step([_entry(pe, s, toks[:15], [14])]).clone()]
    for t in toks[15:]:
        rows.append(eng.step([_entry(pe, s, [t], [0])]).clone())
    eng.free_slot(s)
    models.check(key, dtype, toks, torch.cat(rows), range(14, 255), f"{key} decoding")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["A", "B", "C"])
@pytest.mark.parametrize("portion", [2, 3, 64, 65, 131])
def test_a_prompt_fed_in_portions(pe, models, key, dtype, portion):
    eng = models.engine(key, dtype)
    toks = _tokens(CONFIGS[key]["vocab"], 280, 3)
    s = eng.alloc_slot()
    rows = []
    for lo in range(0, len(toks), portion):
        part = toks[lo:lo + portion]
        rows.append(eng.step([_entry(pe, s, part, range(len(part)))]).clone())
    eng.free_slot(s)
    models.check(key, dtype, toks, torch.cat(rows), range(len(toks)), f"{key} portions of {portion}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", sorted(CONFIGS))
def test_unequal_batches_on_slots_used_again(pe, models, key, dtype):
    """Two batches in a row on the same slots and pages: unequal prompts in one step (among them one token), then one
    token each until the shorter ones have ended; each request against itself alone in the plain implementation."""
    eng = models.engine(key, dtype)
    vocab = CONFIGS[key]["vocab"]
    seen = []
    for batch in range(2):
        plan = [(1, 9), (200, 4), (65, 12), (33, 1), (130, 7)]
        seqs = [_tokens(vocab, p + dec, 100 * batch + i) for i, (p, dec) in enumerate(plan)]
        slots = [eng.alloc_slot() for _ in plan]
        seen.append(sorted(slots))
        got = {}
        out = eng.step([_entry(pe, s, q[:p], [p - 1]) for s, q, (p, dec) in zip(slots, seqs, plan)])
        for i, (p, dec) in enumerate(plan):
            got[i, p - 1] = out[i].clone()
        for step in range(max(dec for _, dec in plan)):
            live = [i for i, (p, dec) in enumerate(plan) if step < dec]
            out = eng.step([_entry(pe, slots[i], [seqs[i][plan[i][0] + step]], [0]) for i in live])
            for r, i in enumerate(live):
                got[i, plan[i][0] + step] = out[r].clone()
                if step == plan[i][1] - 1:
                    eng.free_slot(slots[i])
        assert not eng.cache.live_slots
        for i, (p, dec) in enumerate(plan):
            rows = torch.stack([got[i, j] for j in range(p - 1, p + dec)])
            models.check(key, dtype, seqs[i], rows, range(p - 1, p + dec), f"{key} batch {batch} request {i}")
        eng.cache.check()
    assert seen[0] == seen[1]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("count", [12, 40])
def test_a_decode_batch_of_many(pe, models, dtype, count):
    """More sequences than the weight-streaming products take, inside the captured decode step."""
    key = "B"
    eng = models.engine(key, dtype, max_batch=count, max_cache_tokens=64 * (count + 2))
    vocab = CONFIGS[key]["vocab"]
    seqs = [_tokens(vocab, 3 + i % 13 + 6, 300 + i) for i in range(count)]
    slots = [eng.alloc_slot() for _ in seqs]
    got = {i: [] for i in range(count)}
    out = eng.step([_entry(pe, s, q[:len(q) - 6], [len(q) - 7]) for s, q in zip(slots, seqs)]).clone()
    for i in range(count):
        got[i].append(out[i:i + 1])
    for step in range(6):
        out = eng.step([_entry(pe, s, [q[len(q) - 6 + step]], [0]) for s, q in zip(slots, seqs)]).clone()
        for i in range(count):
            got[i].append(out[i:i + 1])
    for s in slots:
        eng.free_slot(s)
    for i in (0, 5, count - 1):
        n = len(seqs[i])
        models.check(key, dtype, seqs[i], torch.cat(got[i]), range(n - 7, n), f"{key} request {i} of {count}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_model_of_real_layer_sizes_takes_the_many_row_products(pe, models, dtype):
    """1,030 tokens in one step on heads of 128: the products run on the tcgen05 pair kernel (bfloat16), the activation and
    the biases in its epilogue; the last positions against the plain implementation."""
    key = "many rows"
    cfg = {"architecture": "Bobasun", "vocab": 96, "width": 256, "streams": 2, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0},
           "layers": [_layer(_att(4, 2, 128, 128, 0.1, 128, 10000.0, 2.0, mix=True), 512, 1.5),
                      _layer(_att(4, 2, 128, 128, 0.1, 128, 10000.0, 2.0, mix=True), 384, 0.9)]}
    models.add(key, cfg, 91)
    eng = models.engine(key, dtype, max_context_len=1152, max_cache_tokens=64 * 20)
    eng.runtime.large_gemm_min_fill = 0.0
    toks = _tokens(96, 1032, 12)
    if dtype == "bfloat16":
        x = torch.empty(1030, 256, dtype=torch.bfloat16, device=DEV)
        assert all(parts["mixer"].fuses_general_into_product(x, eng.runtime) for parts in eng.model.block_parts)
    positions = list(range(0, 1030, 23)) + [1029]
    s = eng.alloc_slot()
    rows = [eng.step([_entry(pe, s, toks[:1030], positions)]).clone()]
    for t in toks[1030:]:
        rows.append(eng.step([_entry(pe, s, [t], [0])]).clone())
    eng.free_slot(s)
    models.check(key, dtype, toks, torch.cat(rows), positions + [1030, 1031], key)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(pe, models, dtype):
    """``Engine.generate`` with unequal prompts: every generated token must be the plain implementation's best token
    for the sequence so far, or within rounding of it."""
    key = "A"
    eng = models.engine(key, dtype)
    prompts = [_tokens(CONFIGS[key]["vocab"], n, 50 + n) for n in (1, 17, 64, 140)]
    results = eng.generate(prompts, pe.SamplingParams.greedy_params(max_tokens=12))
    for p, r in zip(prompts, results):
        assert len(r.token_ids) == 12
        ref = models.ref(key, p + r.token_ids)
        scale = float(ref.abs().max())
        for j, tok in enumerate(r.token_ids):
            row = ref[len(p) - 1 + j]
            margin = 2 * TOL[dtype] * scale
            if dtype == "bfloat16":      # a logit moves by several times its position's root-mean-square rounding error
                noise = models.noise(key, p + r.token_ids)
                margin = 8.0 * max(float(noise[len(p) - 1 + j]), float(noise.mean()))
            assert float(row.max() - row[tok]) <= margin, (dtype, len(p), j)
    assert not eng.cache.live_slots


def test_a_model_folder_written_at_random_loads_and_runs(pe, tmp_path, capsys):
    """config.json and safetensors through the loader, against the plain implementation on the same file; then the command
    line on the same folder."""
    from importlib import import_module

    from safetensors.torch import load_file

    cfg = pe.BobasunConfig.from_dict(CONFIGS["A"])
    folder = pe.write_random_model(str(tmp_path / "m"), cfg, seed=4)
    assert pe.load_config(folder) == cfg
    eng = pe.Engine(folder, dtype="float32", max_context_len=256, max_cache_tokens=512, max_batch=2)
    w = {k: v.float() for k, v in load_file(folder + "/model.safetensors").items()}
    toks = _tokens(131, 90, 8)
    s = eng.alloc_slot()
    got = eng.step([_entry(pe, s, toks, range(90))]).clone()
    eng.free_slot(s)
    assert rel_err(got.cpu(), plain.forward(CONFIGS["A"], w, toks).float()) < TOL["float32"]
    cli = import_module("pytorch-engine_b200.cli")
    argv = ["--model", folder, "--dtype", "fp32", "--max-tokens", "6", "--temperature", "0", "--json"]
    for n in (3, 40):
        argv += ["--prompt-ids", ",".join(map(str, toks[:n]))]
    assert cli.main(argv) == 0
    out = sorted((json.loads(x) for x in capsys.readouterr().out.splitlines() if x.startswith("{")), key=lambda r: r["request"])
    for r, n in zip(out, (3, 40)):
        ref = plain.forward(CONFIGS["A"], w, toks[:n] + r["token_ids"])
        for j, tok in enumerate(r["token_ids"]):
            assert float(ref[n - 1 + j].max() - ref[n - 1 + j][tok]) <= 1e-4 * float(ref.abs().max())
