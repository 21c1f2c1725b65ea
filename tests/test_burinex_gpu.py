"""The Burinex architecture on the engine against the plain implementation in ``plain_burinex.py``: mechanisms at kernel level
with inputs made so that a fault shows, every mechanism alone as a one-layer model, then whole models: prompts, token-by-token
decoding, prompts in portions, unequal batches, slots and pages used again, long decoding, generation through the entry point."""
import copy
import json
import math

import pytest
import torch

import plain_burinex as plain
from conftest import rel_err

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64
TOL = {"float32": 3e-5, "bfloat16": 2e-2}
# a gap between two experts' router logits below which a bfloat16 rounding may choose otherwise
CLOSE_CALL = 0.05


def _att(heads, kv, dim, vdim, scale, temp=None):
    d = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        d["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": d}


def _lat(heads, dim, rot_dim, vdim, rank, q_rank, scale, window=None, dims=None, base=10000.0, scaling=None):
    d = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale}
    if window:
        d["mask"] = {"size": window}
    if rot_dim:
        d["rot"] = {"base": base, "dims": rot_dim if dims is None else dims}
        if scaling:
            d["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": d}


def _lig(heads, dim, vdim, decay):
    assert len(decay) == heads
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}}


def _moe(experts, top, ff, shared=None):
    d = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def _with(mixer, mlp=None):
    return dict(mixer, mlp=mlp)


# The tests' own models.  A: nothing is a multiple of 8 anywhere (no kernel may take its 16-byte paths), a window that is no
# multiple of a page, a part of the rotated features turned, no shared expert in one layer, no feed-forward in another, no
# temperature in one.  B: sizes that the tensor-core kernels take whole, a window longer than a page, all experts chosen in one
# layer.  C: sizes that run in padded tiles, a window of exactly a page and one of two positions, a state of 136 rows, one head,
# one expert, a temperature that changes at every position, no cap on the logits.  D: a window longer than every sequence, none,
# no rotated part, a decay of one and one of nearly nothing, many experts.
CONFIGS = {
    "A": {"architecture": "Burinex", "vocab": 131, "width": 54, "norm": {"eps": 2e-5}, "postln_alpha": 1.7, "logit_softcap": 12.0,
          "layers": [_with(_lig(3, 10, 14, [0.4, 0.9, 0.99]), _moe(5, 2, 22, 13)),
                     _with(_lat(3, 10, 6, 9, 21, 19, 0.4, 37, 4, 60.0, (3.0, 32, 4.0, 1.0)), _moe(7, 3, 11)),
                     _with(_att(6, 2, 7, 11, 0.5, (0.35, 29))), _with(_att(3, 3, 5, 6, 0.6), _moe(3, 1, 17, 9))]},
    "B": {"architecture": "Burinex", "vocab": 224, "width": 128, "norm": {"eps": 1e-6}, "postln_alpha": 2.5, "logit_softcap": 20.0,
          "layers": [_with(_att(8, 2, 64, 64, 0.1, (0.2, 50)), _moe(8, 2, 64, 128)),
                     _with(_lat(6, 48, 64, 64, 128, 96, 0.1, 100, 64, 10000.0, (4.0, 256, 16.0, 1.0)), _moe(4, 4, 32, 64)),
                     _with(_lig(4, 64, 64, [0.7, 0.95, 0.99, 0.999]), _moe(8, 1, 96, 32)),
                     _with(_att(4, 4, 128, 96, 0.08, (0.4, 100)), _moe(6, 2, 64, 64))]},
    "C": {"architecture": "Burinex", "vocab": 90, "width": 72, "norm": {"eps": 1e-5}, "postln_alpha": 1.0,
          "layers": [_with(_lat(5, 24, 8, 16, 40, 48, 0.3, 64, 8, 500.0, (2.0, 64, 8.0, 2.0)), _moe(1, 1, 24, 40)),
                     _with(_att(2, 1, 72, 40, 0.15, (0.5, 1))),
                     _with(_lat(2, 40, 24, 72, 200, 16, 0.15, 2, 16, 2000.0), _moe(6, 2, 16)),
                     _with(_lig(1, 136, 24, [0.97]), _moe(4, 2, 8, 8)), _with(_att(5, 5, 120, 128, 0.1), _moe(2, 1, 56))]},
    "D": {"architecture": "Burinex", "vocab": 75, "width": 48, "norm": {"eps": 3e-6}, "postln_alpha": 4.0, "logit_softcap": 5.0,
          "layers": [_with(_lat(4, 16, 0, 24, 32, 24, 0.3, 5000), _moe(40, 3, 16, 24)),
                     _with(_lig(2, 32, 8, [1.0, 0.01]), _moe(16, 5, 8)),
                     _with(_lat(3, 8, 16, 8, 24, 40, 0.3, None, 16, 300.0, (8.0, 40, 3.0, 1.0)), _moe(9, 2, 24, 16))]},
}
SEEDS = {"A": 31, "B": 32, "C": 33, "D": 34}


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
            cfg = self.pe.BurinexConfig.from_dict(self.configs[key])
            args = dict(dtype=dtype, max_context_len=1024, max_cache_tokens=64 * 40, max_batch=8)
            args.update(kw)
            self.engines[ident] = self.pe.Engine(None, config=cfg, weights={k: v.to(DEV) for k, v in self.w(key).items()}, **args)
        return self.engines[ident]

    def ref(self, key, toks):
        ident = (key, tuple(toks))
        if ident not in self.refs:
            margins = []
            self.refs[ident] = plain.forward(self.configs[key], self.w(key), toks, margins=margins).float()
            self.refs[ident + ("decided",)] = (torch.stack(margins).min(0).values if margins
                                               else torch.full((len(toks),), float("inf"), dtype=F64))
        return self.refs[ident]

    def decided(self, key, toks):
        """Per position: the smallest gap by which any router of the model chose its experts there."""
        self.ref(key, toks)
        return self.refs[(key, tuple(toks), "decided")]

    def noise(self, key, toks):
        """How far rounding to bfloat16 alone moves each position's logits (root mean square over the vocabulary)."""
        ident = (key, tuple(toks), "noise")
        if ident not in self.refs:
            with plain.stored(torch.bfloat16):
                rounded = plain.forward(self.configs[key], self.w(key), toks)
            self.refs[ident] = (rounded - self.ref(key, toks).double()).pow(2).mean(dim=1).sqrt()
        return self.refs[ident]

    def check(self, key, dtype, toks, got, positions, what):
        """float32: every logit within 3e-5 of the largest.  bfloat16: the error is held against what rounding alone does in
        the plain implementation: its median at most twice that (three times for fewer than 30 positions), and at no more than
        one position in twenty (or two) above four times the larger of that position's own figure and the average.  Positions where a router's choice hung on a gap of
        less than CLOSE_CALL are left out: there a rounding may pick another expert, in the engine or in the measure."""
        positions = list(positions)
        ref = self.ref(key, toks)[positions]
        got = got.float().cpu()
        assert got.shape == ref.shape, what
        if dtype == "float32":
            err = rel_err(got, ref)
            assert err < TOL[dtype], f"{what}: error {err:.3e} (limit {TOL[dtype]:.0e})"
            return
        noise = self.noise(key, toks)
        floor = float(noise.median())
        decided = self.decided(key, toks)
        keep = [i for i, p in enumerate(positions) if float(decided[p]) >= CLOSE_CALL]
        if not keep:
            assert len(positions) <= 2, f"{what}: only nearly tied experts"
            return
        assert len(keep) >= len(positions) // 4, f"{what}: too many positions with nearly tied experts"
        rows = [positions[i] for i in keep]
        err = (got[keep].double() - ref[keep].double()).pow(2).mean(dim=1).sqrt()
        limit = (2.0 if len(rows) >= 30 else 3.0) * max(float(noise[rows].median()), floor)
        assert float(err.median()) <= limit, f"{what}: median error {float(err.median()):.3e}, limit {limit:.3e}"
        over = int((err > 4.0 * torch.clamp(noise[rows], min=floor)).sum())
        assert over <= max(2, len(rows) // 20), f"{what}: {over} of {len(rows)} positions beyond four times rounding"


@pytest.fixture(scope="module")
def models(pe):
    return Models(pe)


@pytest.fixture(scope="module")
def ops(pe):
    return pe.kernels.ops


def _entry(pe, slot, toks, want):
    return pe.StepEntry(slot, toks, tuple(want))


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def _status():
    return torch.zeros(4, dtype=torch.int32, device=DEV)


class Paged:
    """Sequences whose rows lie scattered over shuffled pages of a pool that holds junk elsewhere."""

    def __init__(self, lens, heads, dim, dtype, seed=0):
        g = torch.Generator().manual_seed(seed)
        per = [(n + 63) // 64 for n in lens]
        self.num_pages = sum(per) + 4
        order = torch.randperm(self.num_pages, generator=g).tolist()
        self.slots = list(range(len(lens) - 1, -1, -1))
        table = torch.full((len(lens) + 1, max(per) + 1), -1, dtype=torch.int32)
        for b, p in enumerate(per):
            for lp in range(p):
                table[self.slots[b], lp] = order.pop()
        self.pages = (50.0 * torch.randn(self.num_pages, heads, 64, dim, generator=g)).to(dtype).to(DEV)
        self.table, self.seq_slot = table.to(DEV), _i32(self.slots)

    def put(self, b, rows):
        """rows [len, heads, dim] of sequence b into its pages."""
        for lp in range((rows.shape[0] + 63) // 64):
            page, part = int(self.table[self.slots[b], lp]), rows[lp * 64:lp * 64 + 64]
            self.pages[page, :, :part.shape[0]] = part.transpose(0, 1).to(self.pages.dtype).to(DEV)


def _batch(q_lens, pasts):
    """(token_seq, token_pos, seq_qstart, seq_past) of a step, int32 on the device."""
    seq = [b for b, n in enumerate(q_lens) for _ in range(n)]
    pos = [p + j for n, p in zip(q_lens, pasts) for j in range(n)]
    return _i32(seq), _i32(pos), _i32([0] + torch.tensor(q_lens).cumsum(0).tolist()), _i32(list(pasts))


# ---- mechanisms at kernel level -----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,dim", [(5, 50), (3, 72), (70, 1028), (3, 4096), (90, 4096), (2, 9000), (2, 20000)])
def test_norm_behind_the_sum(ops, dtype, n, dim):
    """The stream becomes the norm of alpha times itself plus the scaled output, with a factor per feature and without, with the
    copy for the next sublayer and without; the eps is large enough to show."""
    g = torch.Generator().manual_seed(dim)
    x, y = 0.3 * torch.randn(n, dim, generator=g), (0.2 * torch.randn(n, dim, generator=g)).to(dtype)
    w, s = 1.0 + 0.3 * torch.randn(dim, generator=g), torch.randn(dim, generator=g)
    for scale in (s, None):
        for alpha, eps in ((2.5, 0.05), (1.0, 1e-6)):
            h = alpha * x.double() + y.double() * (1.0 if scale is None else scale.double())
            want = plain.unit(h, eps) * w.double()
            for with_cast in (True, False):
                stream = x.to(DEV)
                cast = torch.full((n, dim), float("nan"), dtype=dtype, device=DEV) if with_cast else None
                ops.rmsnorm_of_sum(stream, y.to(DEV), alpha, None if scale is None else scale.to(DEV), w.to(DEV), eps, cast)
                assert rel_err(stream.cpu(), want) < 2e-6
                if with_cast:
                    assert torch.equal(cast, stream.to(dtype))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,dim,ld", [(5, 50, 61), (3, 72, 200), (400, 1536, 2112), (3, 1536, 2112), (2, 9000, 9000), (2, 20000, 20004)])
def test_norm_of_columns_of_wider_rows(ops, dtype, n, dim, ld):
    g = torch.Generator().manual_seed(dim + n)
    x, w = torch.randn(n, ld, generator=g).to(dtype), 1.0 + 0.3 * torch.randn(dim, generator=g)
    out = torch.empty(n, dim, dtype=dtype, device=DEV)
    ops.rmsnorm(x.to(DEV)[:, :dim], w.to(DEV), out, 0.02)
    assert rel_err(out.cpu(), plain.unit(x[:, :dim].double(), 0.02) * w.double()) < (2e-6 if dtype == torch.float32 else 6e-3)


def test_capped_logits(ops):
    x = torch.linspace(-300, 300, 1001).to(DEV)
    y = x.clone()
    ops.softcap_(y, 7.5, 0.5)
    assert (y.double().cpu() - 7.5 * torch.tanh(0.5 * x.double().cpu() / 7.5)).abs().max() < 2e-6
    assert float(y.abs().max()) <= 7.5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 16, 24), (3, 1, 7, 5), (6, 3, 64, 80), (1, 1, 8, 8), (32, 8, 128, 128), (5, 5, 200, 16)])
@pytest.mark.parametrize("rotation", [None, "halves", "pairs"])
def test_one_norm_over_all_heads_temperature_and_append(ops, dtype, H, G, d, dv, rotation):
    """Queries and keys normed over their whole rows (one head far larger than the others, so that a norm per head shows), the
    temperature at positions around its steps, keys and values in their pages, the rest of a started page cleared; few tokens
    and many, from the middle of a page; with and without weights, temperature and rotation."""
    lens, q_lens = [300, 65, 129, 1], [290, 1, 2, 1]
    if H > 8:
        lens, q_lens = [70, 65, 129, 1], [9, 1, 2, 1]
    n, pasts = sum(q_lens), [a - b for a, b in zip(lens, q_lens)]
    g = torch.Generator().manual_seed(H + d)
    cols = (H + G) * d + G * dv
    extra = 8 if cols % 8 == 0 else 3
    x = torch.randn(n, cols + extra, generator=g)
    x[:, :d] *= 6.0
    x[:, H * d:H * d + d] *= 0.1
    x = x.to(dtype)
    qw, kw = 1.0 + 0.3 * torch.randn(H * d, generator=g), 1.0 + 0.3 * torch.randn(G * d, generator=g)
    rot = 0 if rotation is None else d // 2 // 2 * 2
    cos = sin = None
    if rot:
        ang = torch.arange(320, dtype=F64)[:, None] * 50.0 ** (-2.0 * torch.arange(rot // 2, dtype=F64) / rot)
        cos, sin = torch.cos(ang).float().to(DEV), torch.sin(ang).float().to(DEV)
    seq, pos, qstart, past = _batch(q_lens, pasts)
    p = pos.cpu().long()
    for weights in (True, False):
        for temp in ((0.7, 16), None):
            K, V = Paged(lens, G, d, dtype, seed=1), Paged(lens, G, dv, dtype, seed=1)
            row = x.to(DEV)
            st = _status()
            ops.qkv_row_norm_append(row, n, H, G, d, dv, qw.to(DEV) if weights else None, kw.to(DEV) if weights else None, 0.01, temp,
                                    cos, sin, rot, rotation == "pairs", seq, pos, K.seq_slot, qstart, K.table, K.num_pages, K.pages,
                                    V.pages, True, st)
            assert st.tolist()[0] == 0
            q, k = x[:, :H * d].double(), x[:, H * d:(H + G) * d].double()
            if weights:
                q, k = plain.unit(q, 0.01) * qw.double(), plain.unit(k, 0.01) * kw.double()
            if temp:
                q = q * (1.0 + temp[0] * torch.log(((p + 1) // temp[1]).double() + 1.0))[:, None]
            q, k = q.view(n, H, d), k.view(n, G, d)
            if rot:
                c, s = torch.cos(ang)[p][:, None, :], torch.sin(ang)[p][:, None, :]
                for t in (q, k):
                    a, b = (t[..., 0:rot:2], t[..., 1:rot:2]) if rotation == "pairs" else (t[..., :rot // 2], t[..., rot // 2:rot])
                    a0, b0 = a.clone(), b.clone()
                    a.copy_(a0 * c - b0 * s)
                    b.copy_(b0 * c + a0 * s)
            tol = 1e-5 if dtype == torch.float32 else 6e-3
            assert rel_err(row[:, :H * d].cpu(), q.reshape(n, H * d)) < tol
            assert torch.equal(row[:, cols:].cpu(), x[:, cols:])
            got_k, got_v = K.pages.cpu(), V.pages.cpu()
            table = K.table.cpu()
            scale = float(k.abs().max())
            for t in range(n):
                b, off = int(seq[t]), int(p[t]) % 64
                page = int(table[K.slots[b], int(p[t]) // 64])
                assert (got_k[page, :, off].double() - k[t]).abs().max() < tol * scale
                assert torch.equal(got_v[page, :, off], x[t, (H + G) * d:cols].view(G, dv))
                if t == n - 1 or int(seq[t + 1]) != b:
                    rest_k, rest_v = got_k[page, :, off + 1:], got_v[page, :, off + 1:]
                    if q_lens[b] > 1 or off == 0:
                        assert rest_k.numel() == 0 or (float(rest_k.abs().max()) == 0.0 and float(rest_v.abs().max()) == 0.0)


@pytest.mark.parametrize("d,dv", [(8, 8), (24, 20), (64, 48), (128, 64), (136, 12), (40, 100), (300, 8), (100, 260), (16, 600), (7, 3)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_lightning_recurrence_whole_chunked_in_steps_and_on_kept_state(ops, d, dv, dtype):
    """Whole sequences (short: one go; long: chunks side by side) against the same sequences cut into steps of 1, 3 and many
    tokens, two sequences of unequal length on slots whose neighbours hold other state, against the plain recurrence; decays
    from nearly nothing to one, and none at all."""
    decay = [0.0, 0.5, 0.99, 1.0]
    heads = len(decay)
    g = torch.Generator().manual_seed(d + dv)
    lens = [300, 41]
    cols = heads * (2 * d + dv)
    xs = [torch.randn(n, cols + 8, generator=g).to(dtype) for n in lens]          # q | k | v are columns of wider rows
    want = []
    for x in xs:
        z = torch.nn.functional.silu(x[:, :cols].double())
        q, k, v = z[:, :heads * d].view(-1, heads, d), z[:, heads * d:2 * heads * d].view(-1, heads, d), z[:, 2 * heads * d:].view(-1, heads, dv)
        S, y = torch.zeros(heads, d, dv, dtype=F64), torch.zeros(len(x), heads, dv, dtype=F64)
        for t in range(len(x)):
            S = torch.tensor(decay, dtype=F64)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
            y[t] = torch.einsum("hij,hi->hj", S, q[t])
        want.append(y.reshape(len(x), heads * dv))
    dec = torch.tensor(decay, device=DEV)
    logs = torch.tensor([math.log(x) if x else -math.inf for x in decay], device=DEV)
    st = _status()
    for cuts in ([300], [1, 3, 1, 200, 95]):
        S = torch.randn(5, heads, d, dv, device=DEV)                              # slots 0, 2, 4 keep what they hold
        before = S.clone()
        S[1].zero_()
        S[3].zero_()
        got, at = [[], []], [0, 0]
        for step in cuts:
            live = [b for b in range(2) if at[b] < lens[b]]
            q = [min(step, lens[b] - at[b]) for b in live]
            qstart = _i32([0] + torch.tensor(q).cumsum(0).tolist())
            x = torch.cat([xs[b][at[b]:at[b] + n] for b, n in zip(live, q)]).to(DEV)
            y = torch.full((sum(q), heads * dv), float("nan"), device=DEV)
            chunk, max_chunks, scratch = 0, 1, None
            if max(q) > 128:
                chunk, max_chunks = 64, -(-max(q) // 64)
                scratch = torch.full((ops.ssd_scratch_floats(len(live), heads, d, dv, max_chunks),), float("nan"), device=DEV)
            ops.lightning_recurrence(x[:, :cols], dec, logs, y, S, _i32([3 - 2 * b for b in live]), qstart, len(live), max(q), heads, d,
                                     dv, st, chunk, max_chunks, scratch)
            for b, n, lo in zip(live, q, qstart.tolist()):
                got[b].append(y[lo:lo + n].cpu())
                at[b] += n
        for b in range(2):
            have = torch.cat(got[b]).double().view(-1, heads, dv)
            ref = want[b].view(-1, heads, dv)
            for h in range(heads):                     # each head by its own scale: one of them holds far more than the others
                err = (have[:, h] - ref[:, h]).abs().max() / ref[:, h].abs().max()
                assert err < 2e-5, (d, dv, cuts, b, h, float(err))
        assert torch.equal(S[[0, 2, 4]], before[[0, 2, 4]])
    assert st.tolist()[0] == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,width,parts", [(5, 50, 1), (3, 72, 3), (400, 2048, 1), (3, 4096, 1), (2, 12000, 1), (6, 96, 6)])
def test_norm_then_gate_and_gate_then_norm(ops, dtype, n, width, parts):
    g = torch.Generator().manual_seed(width)
    y, z, w = torch.randn(n, width, generator=g), torch.randn(n, width + 12, generator=g).to(dtype), 1.0 + 0.3 * torch.randn(width, generator=g)
    zz = z[:, 12:].double()
    for first in (True, False):
        out = torch.empty(n, width, dtype=dtype, device=DEV)
        ops.gated_part_norm(y.to(DEV), z.to(DEV)[:, 12:], w.to(DEV), 0.02, out, parts, gate_first=first)
        v = y.double() * (zz * torch.sigmoid(zz) if first else 1.0)
        v = plain.unit(v.view(n, parts, width // parts), 0.02).view(n, width) * w.double()
        assert rel_err(out.cpu(), v if first else v * torch.sigmoid(zz)) < (3e-6 if dtype == torch.float32 else 6e-3), first


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,E,top,H,ff", [(1, 5, 2, 40, 24), (4, 6, 6, 50, 7), (3, 3, 1, 64, 32), (40, 12, 3, 64, 48), (9, 4, 2, 128, 64)])
def test_experts_weighted_on_their_input(pe, dtype, n, E, top, H, ff):
    """Against each chosen expert run on its weighted input: few tokens and many, one expert and all; sigmoid scores near zero
    and one, so that a weight on the output instead of the input shows."""
    class Ctx:
        def buffer(self, name, shape, dt):
            return torch.full(shape, float("nan"), device=DEV).to(dt) if dt.is_floating_point else torch.zeros(shape, dtype=dt, device=DEV)

    g = torch.Generator().manual_seed(n + E)
    rt = pe.parts.Runtime(torch.device(DEV), dtype)
    w = {"router": 0.5 * torch.randn(E, H, generator=g)}
    for e in [f"e{i}" for i in range(E)] + ["shared"]:
        w.update({f"{e}.gate": torch.randn(ff, H, generator=g) / H ** 0.5, f"{e}.up": torch.randn(ff, H, generator=g) / H ** 0.5,
                  f"{e}.down": torch.randn(H, ff, generator=g) / ff ** 0.5})
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    h = torch.randn(n, H, generator=g).to(torch.bfloat16).float()
    params = {"hidden": H, "n_experts": E, "n_identity": 0, "top": top, "intermediate": ff, "activation": "silu",
              "choice": "sigmoid_groups", "weight_on": "input", "shared": {"intermediate": ff}}
    cls = pe.parts.lookup("feed_forward", "routed_experts")
    part = cls(params, {k: v.to(DEV) for k, v in w.items()}, rt)
    got = part.forward(h.to(DEV, dtype), Ctx()).double().cpu()
    spec = {"router": {"experts": E, "top": top}, "expert": {"ff": ff}, "shared": {"ff": ff}}
    want = plain.moe_ff(h.double(), spec, {f"x.{k}": v.double() for k, v in w.items()}, "x")
    assert rel_err(got, want) < (3e-6 if dtype == torch.float32 else 1.5e-2)
    rt = pe.parts.Runtime(torch.device(DEV), dtype)
    other = cls(dict(params, weight_on="output"), {k: v.to(DEV) for k, v in w.items()}, rt).forward(h.to(DEV, dtype), Ctx())
    assert rel_err(other.double().cpu(), want) > 5e-2


def test_the_largest_score_is_chosen_where_the_sigmoid_is_one_or_nothing_in_float32(ops):
    """Logits so large (or so far below zero) that float32 cannot tell their sigmoids apart, and ordinary ones."""
    for base in (25.0, 0.0, -120.0):
        logits = base + torch.tensor([[0.0, 0.002, -0.5, 0.001, 0.5, 0.499]]).repeat(3, 1)
        logits[1, 0], logits[2, 3] = base + 0.75, base + 0.75
        chosen = torch.empty(3, 2, dtype=torch.int32, device=DEV)
        weight = torch.empty(3, 2, device=DEV)
        ops.moe_route_sigmoid_groups(logits.to(DEV), 2, 1, 1, chosen, weight)
        assert chosen.tolist() == [[4, 5], [0, 4], [3, 4]]
        want = torch.sigmoid(logits.double().gather(1, chosen.cpu().long()))
        assert (weight.double().cpu() - want).abs().max() < 1e-6


def _latent_attend(ops, kernel, decode, q, lens, q_lens, nh, row, r, scale, pg, window, sinks, even=True):
    """The step's output rows ``[n, nh * r]`` and the split results of both ways to cut a decode into ranges."""
    n, dtype = sum(q_lens), pg.pages.dtype
    seq, pos, qstart, past = _batch(q_lens, [a - b for a, b in zip(lens, q_lens)])
    out = torch.full((n, nh * r), float("nan"), dtype=dtype, device=DEV)
    st = _status()
    args = (decode, q.to(dtype).to(DEV), out, len(lens), max(q_lens), nh)
    where = (qstart, past, pg.seq_slot, pg.table, pg.num_pages)
    sinks = None if sinks is None else sinks.to(DEV)
    if kernel == "tensor cores":
        split, splits, floor, scratch = 0, 0, 0, None
        if decode:
            split, splits, floor = (0, 3, 0) if even else (64, -(-max(lens) // 64), 0)
            scratch = torch.full((ops.attention_generic_scratch_floats(len(lens), nh, r, splits),), float("nan"), device=DEV)
        ops.attention_latent(*args, row, r, scale, *where, pg.pages, scratch, split, splits, st, min_range_keys=floor, window=window,
                             sinks=sinks)
    else:
        splits = -(-max(lens) // 64) if decode else 0
        scratch = torch.full((ops.attention_generic_scratch_floats(len(lens), nh, r, splits),), float("nan"), device=DEV) if decode else None
        ops.attention_generic_masked(*args, 1, row, r, scale, *where, pg.pages, pg.pages, scratch, 64, splits, st, v_ld=row,
                                     window=window, sinks=sinks)
    assert st.tolist()[0] == 0
    return out.double().cpu()


@pytest.mark.parametrize("kernel,dtype", [("float32 arithmetic", torch.float32), ("float32 arithmetic", torch.bfloat16),
                                          ("tensor cores", torch.bfloat16)])
@pytest.mark.parametrize("row,r,nh,window", [(96, 64, 5, 40), (48, 40, 3, 64), (128, 128, 17, 1), (136, 72, 16, 200), (384, 384, 2, 65),
                                             (576, 512, 20, 130), (232, 200, 4, 0), (64, 8, 6, 63)])
def test_cached_rows_under_a_window_with_sinks(ops, kernel, dtype, row, r, nh, window):
    """Prompts that start at a page's border, in its middle and at position 0, one token, and decoding with more heads than one
    block takes, sinks from far below the scores to far above; against the plain softmax on the same inputs."""
    if kernel == "tensor cores":
        assert ops.attention_latent_supported(dtype, row, r)
    lens, q_lens = [500, 65, 300, 192], [130, 65, 1, 64]
    g = torch.Generator().manual_seed(row + nh)
    pg = Paged(lens, 1, row, dtype, seed=2)
    rows = [torch.randn(n, 1, row, generator=g) for n in lens]
    for b in range(len(lens)):
        pg.put(b, rows[b])
    scale = 1.5 / math.sqrt(row)
    sinks = torch.linspace(-30, 12, nh)
    for decode, ql in ((False, q_lens), (True, [1] * len(lens))):
        q = torch.randn(sum(ql), nh * row, generator=g)
        for sk in (sinks, None):
            for even in (True, False) if decode else (True,):
                out = _latent_attend(ops, kernel, decode, q, lens, ql, nh, row, r, scale, pg, window, sk, even)
                at = 0
                for b, (L, m) in enumerate(zip(lens, ql)):
                    keys = rows[b][:, 0].to(dtype).double()
                    pos, j = torch.arange(L - m, L)[:, None], torch.arange(L)[None, :]
                    seen = (j <= pos) & ((pos - j < window) if window else True)
                    for h in range(nh):
                        s = q[at:at + m, h * row:(h + 1) * row].to(dtype).double() @ keys.T * scale
                        want = plain.sink_softmax(s, seen, -math.inf if sk is None else sk[h].double()) @ keys[:, :r]
                        err = float((out[at:at + m, h * r:(h + 1) * r] - want).abs().max())
                        assert err < (2e-5 if dtype == torch.float32 else 2e-2), (decode, b, h, err)
                    at += m


@pytest.mark.parametrize("kernel", ["float32 arithmetic", "tensor cores"])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window", [1, 2, 40, 63, 64, 65, 130])
def test_keys_just_inside_and_just_outside_the_window(ops, kernel, decode, window):
    """One key matches the query far better than all others: at the window's oldest position the output is its row, one
    position further back it must not be seen and the sink, which stands above the rest, takes the weight.  The query sits so
    that the edge falls before, on and behind page borders; a prompt's queries are the last five of the sequence."""
    row, r, nh = 24, 16, 3
    dtype = torch.float32 if kernel == "float32 arithmetic" else torch.bfloat16
    for n in sorted({window + 1, 64, 65, 128, 129, 127 + window, 128 + window, 300}):
        i = n - 1
        lo = max(0, i - window + 1)
        for target in {lo, lo - 1, i}:
            if target < 0:
                continue
            g = torch.Generator().manual_seed(n + target)
            keys = torch.randn(n, 1, row, generator=g)
            keys[:, :, 20] = 0.0
            keys[target, :, 20] = 1.0
            pg = Paged([n], 1, row, dtype, seed=n)
            pg.put(0, keys)
            nq = 1 if decode else min(5, n)
            q = torch.zeros(nq, nh * row)
            q.view(nq, nh, row)[:, :, 20] = 100.0
            for even in (True, False) if decode else (True,):
                out = _latent_attend(ops, kernel, decode, q, [n], [nq], nh, row, r, 0.5, pg, window, torch.full((nh,), 25.0), even)
                got = out[-1].view(nh, r)
                want = keys[target, 0, :r].to(dtype).double() if target >= lo else torch.zeros(r, dtype=F64)
                assert (got - want).abs().max() < (1e-4 if dtype == torch.float32 else 2e-2), (n, target, lo)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_in_a_prompt_and_decoded(pe, models, dtype):
    """One attention layer whose last query has one key that stands out, far back among hundreds: the token at position 3 alone
    has the key feature that the last token asks for."""
    key = "far " + dtype
    cfg = {"architecture": "Burinex", "vocab": 64, "width": 32, "norm": {"eps": 1e-5}, "postln_alpha": 0.3,
           "layers": [_with(_att(2, 1, 16, 24, 1.0, (0.4, 64)))]}
    models.add(key, cfg, 5)
    w = models.w(key)
    w["embed"][:, :2] = 0.0
    w["embed"][7, 0] = 6.0                                   # the token that is looked for
    w["embed"][5, 1] = 6.0                                   # the token that looks
    for n in ("q", "k"):
        w[f"l0.mix.{n}"] *= 0.1
    w["l0.mix.q"][12] = w["l0.mix.q"][28] = 0.0
    w["l0.mix.k"][12] = 0.0
    w["l0.mix.q"][12, 1] = w["l0.mix.q"][28, 1] = 4.0
    w["l0.mix.k"][12, 0] = 4.0
    w["l0.mix.q.norm"].fill_(1.0)
    w["l0.mix.k.norm"].fill_(1.0)
    toks = [t if t not in (5, 7) else 8 for t in _tokens(64, 500, 5)]
    toks[3], toks[-1] = 7, 5
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
    assert rel_err(plain.forward(cfg, w, other)[499:].float(), models.ref(key, toks)[499:]) > 5e-2


# ---- every mechanism alone, as a model of one layer -------------------------------------------------------------------
_TINY = _lig(1, 8, 8, [0.9])
ALONE = {
    "attention": [_with(_att(4, 2, 12, 20, 0.4, (0.5, 17)))],
    "attention without temperature": [_with(_att(4, 1, 24, 16, 0.5))],
    "attention on tensor cores": [_with(_att(8, 2, 64, 48, 0.12, (0.3, 32)))],
    "attention with keys beyond 64": [_with(_att(4, 2, 96, 64, 0.1, (0.3, 40)))],
    "latent": [_with(_lat(3, 12, 8, 20, 28, 18, 0.4, 30, 8, 200.0, (4.0, 32, 8.0, 1.0)))],
    "latent without a window": [_with(_lat(3, 12, 4, 8, 20, 10, 0.4, None, 4, 200.0))],
    "latent without rotation": [_with(_lat(2, 16, 0, 8, 24, 16, 0.4, 50))],
    "latent on tensor cores": [_with(_lat(6, 24, 16, 32, 48, 40, 0.2, 70, 16, 5000.0, (2.0, 100, 8.0, 2.0)))],
    "lightning": [_with(_lig(4, 12, 20, [0.3, 0.8, 0.97, 0.999]))],
    "experts": [_with(_TINY, _moe(7, 2, 24, 40))],
    "experts, one of many": [_with(_TINY, _moe(64, 1, 16))],
    "experts, wide": [_with(_TINY, _moe(4, 3, 128, 64))],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_one_mechanism_alone_whole_and_token_by_token(pe, models, name, dtype):
    key = "alone " + name
    cfg = {"architecture": "Burinex", "vocab": 90, "width": 64, "norm": {"eps": 1e-5}, "postln_alpha": 1.3, "logit_softcap": 15.0,
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


# ---- whole models -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", sorted(CONFIGS))
def test_whole_prompt_and_its_first_tokens(pe, models, key, dtype):
    eng = models.engine(key, dtype)
    toks = _tokens(CONFIGS[key]["vocab"], 300, 1)
    s = eng.alloc_slot()
    got = eng.step([_entry(pe, s, toks, range(300))]).clone()
    eng.free_slot(s)
    models.check(key, dtype, toks, got, range(300), f"{key} whole prompt")
    s = eng.alloc_slot()                               # a prompt of one token, then of two, on the slot that was just freed
    rows = [eng.step([_entry(pe, s, toks[:1], [0])]).clone()]
    eng.free_slot(s)
    s = eng.alloc_slot()
    rows.append(eng.step([_entry(pe, s, toks[:2], [1])]).clone())
    eng.free_slot(s)
    models.check(key, dtype, toks, torch.cat(rows), range(2), f"{key} first tokens on a used slot")
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


def test_pages_behind_the_window_are_given_back_and_used_again(pe, models):
    """A model of window layers only holds the window's pages however long its sequence grows, and a second sequence that takes
    the pages the first one gave back changes nothing for it."""
    key = "window pages"
    cfg = {"architecture": "Burinex", "vocab": 70, "width": 40, "norm": {"eps": 1e-5}, "postln_alpha": 1.5,
           "layers": [_with(_lat(2, 8, 8, 8, 16, 16, 0.4, 70, 8, 100.0)), _with(_lig(2, 8, 8, [0.9, 0.99]))]}
    models.add(key, cfg, 61)
    eng = models.engine(key, "float32", max_context_len=512, max_cache_tokens=64 * 6, max_batch=2)
    a, b = _tokens(70, 330, 1), _tokens(70, 150, 2)
    s = eng.alloc_slot()
    rows_a = [eng.step([_entry(pe, s, a[:130], range(130))]).clone()]
    rows_b, t = [], None
    for i, tok in enumerate(a[130:]):
        entries = [_entry(pe, s, [tok], [0])]
        if i == 60:
            t = eng.alloc_slot()
            rows_b.append(eng.step([_entry(pe, t, b[:100], range(100))]).clone())
        if t is not None and len(rows_b) - 1 < 50:
            entries.append(_entry(pe, t, [b[99 + len(rows_b)]], [0]))
        out = eng.step(entries).clone()
        rows_a.append(out[:1])
        if len(entries) == 2:
            rows_b.append(out[1:])
        held = sum(p >= 0 for p in eng.cache.groups[0].pages_of_slot[s])
        assert held <= 3, (i, held)
    models.check(key, "float32", a, torch.cat(rows_a), range(330), "the long one")
    models.check(key, "float32", b, torch.cat(rows_b), range(150), "the one on its pages")
    eng.free_slot(s)
    eng.free_slot(t)
    eng.cache.check()
    assert eng.free_pages() == 6


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
def test_many_rows_of_larger_layers(pe, models, dtype):
    """1,030 tokens in one step: the many-row products, the experts' library product, sixteen chunks of the recurrence; chosen
    positions against the plain implementation."""
    key = "many rows"
    cfg = {"architecture": "Burinex", "vocab": 96, "width": 256, "norm": {"eps": 1e-5}, "postln_alpha": 2.0, "logit_softcap": 30.0,
           "layers": [_with(_lat(8, 64, 32, 64, 160, 192, 0.1, 300, 32, 10000.0, (4.0, 512, 16.0, 1.0)), _moe(6, 2, 128, 256)),
                      _with(_lig(4, 64, 128, [0.8, 0.97, 0.995, 0.9995])), _with(_att(6, 2, 128, 128, 0.08, (0.1, 200)), _moe(8, 1, 64, 64))]}
    models.add(key, cfg, 91)
    eng = models.engine(key, dtype, max_context_len=1152, max_cache_tokens=64 * 20)
    eng.runtime.large_gemm_min_fill = 0.0
    toks = _tokens(96, 1032, 12)
    positions = list(range(0, 1030, 23)) + [1029]
    s = eng.alloc_slot()
    rows = [eng.step([_entry(pe, s, toks[:1030], positions)]).clone()]
    for t in toks[1030:]:
        rows.append(eng.step([_entry(pe, s, [t], [0])]).clone())
    eng.free_slot(s)
    models.check(key, dtype, toks, torch.cat(rows), positions + [1030, 1031], key)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["A", "B"])
def test_greedy_generation_through_the_entry_point(pe, models, key, dtype):
    """``Engine.generate`` with unequal prompts: every generated token must be the plain implementation's best token for the
    sequence so far, or within rounding of it (in bfloat16 at one position in ten another expert may have been chosen)."""
    eng = models.engine(key, dtype)
    prompts = [_tokens(CONFIGS[key]["vocab"], n, 50 + n) for n in (1, 17, 64, 140)]
    results = eng.generate(prompts, pe.SamplingParams.greedy_params(max_tokens=12))
    missed = 0
    for p, r in zip(prompts, results):
        assert len(r.token_ids) == 12
        seq = p + r.token_ids
        ref = models.ref(key, seq)
        for j, tok in enumerate(r.token_ids):
            at = len(p) - 1 + j
            margin = 2 * TOL[dtype] * float(ref.abs().max())
            if dtype == "bfloat16":      # a logit moves by several times its position's root-mean-square rounding error
                noise = models.noise(key, seq)
                margin = 8.0 * max(float(noise[at]), float(noise.mean()))
            missed += float(ref[at].max() - ref[at][tok]) > margin
    assert missed <= (0 if dtype == "float32" else 4), missed
    assert not eng.cache.live_slots


def test_a_model_folder_written_at_random_loads_and_runs(pe, tmp_path, capsys):
    """config.json and safetensors through the loader, against the plain implementation on the same file; then the command
    line on the same folder."""
    from importlib import import_module

    from safetensors.torch import load_file

    cfg = pe.BurinexConfig.from_dict(CONFIGS["A"])
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
