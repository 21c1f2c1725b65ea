"""The Burinex decoder written out plainly and slowly in PyTorch, one function per mechanism, for the tests.

It shares no code with the package: it reads a configuration as a plain dict (the keys of ``config.json``) and weights
as a dict of tensors by checkpoint name, and computes everything in the dtype it is given (float64 by default), one
whole sequence at a time, with no cache and no state carried from call to call.

Notation: ``x`` is the residual stream ``[T, width]``; ``unit(x) = x / sqrt(mean(x^2) + eps)``.

    layer:      x <- unit(alpha x + s1 * mixer(x)) * w1 ;  x <- unit(alpha x + s2 * ff(x)) * w2      (s: one factor a feature)
    attention:  q, k divided by their root mean square over all heads together, times a weight; q times
                1 + coef ln(floor((p + 1) / every) + 1); causal softmax over grouped heads whose denominator has one more
                term e^0; each head times sigmoid((W_g h)_head); W_o
    latent:     q = W_uq (unit(W_dq h) * w) ; [low | r] = W_dkv h ; c = unit(low) * w ; k = [W_uk c | turn(r)] ; v = W_uv c ;
                softmax over the last ``size`` positions whose denominator has one more term e^sink a head; W_o
    lightning:  q, k, v = silu(W h) ; per head S <- decay S + k v^T ; o = S^T q ; W_o (unit(all heads) * w * sigmoid(W_g h))
    ff:         s = sigmoid(R h) ; the ``top`` largest ; sum of expert(s h) + shared(h) ; expert(z) = D (silu(G z) * (U z))
    output:     cap tanh(W unit(x) w / cap)
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch
import torch.nn.functional as F

# ``STORE``: None, or a 16-bit dtype in which the results of matrix products are rounded (and brought back), at about
# the places where an engine that runs in that dtype rounds: the measure against which a 16-bit run is judged.
STORE = None


class stored:
    def __init__(self, dtype):
        self.dtype = dtype

    def __enter__(self):
        global STORE
        self.before, STORE = STORE, self.dtype

    def __exit__(self, *exc):
        global STORE
        STORE = self.before


def st(x: torch.Tensor) -> torch.Tensor:
    return x if STORE is None else x.to(STORE).to(x.dtype)


def lin(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return st(x @ w.T)


def unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


# ---- feed-forward ---------------------------------------------------------------------------------------------
def gated(z: torch.Tensor, w: Dict[str, torch.Tensor], p: str, factor: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``D (silu(G z f) * (U z f))`` with a factor ``f`` per row (an engine applies it behind the rounded products)."""
    g, u = lin(z, w[f"{p}.gate"]), lin(z, w[f"{p}.up"])
    if factor is not None:
        g, u = g * factor[:, None], u * factor[:, None]
    return lin(st(F.silu(g) * u), w[f"{p}.down"])


def router_choice(logits: torch.Tensor, top: int, margins: Optional[list] = None):
    """``logits [T, E]`` -> (chosen [T, top], their sigmoid scores).  ``margins`` (a list) gets one tensor ``[T]``: the gap, in
    logits, between the last chosen output and the best one left out."""
    E = logits.shape[1]
    ranked = logits.topk(min(top + 1, E), dim=-1)
    if margins is not None:
        margins.append(ranked.values[:, top - 1] - ranked.values[:, top] if top < E
                       else torch.full((logits.shape[0],), float("inf"), dtype=logits.dtype))
    return ranked.indices[:, :top], torch.sigmoid(ranked.values[:, :top])


def moe_ff(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor], p: str, margins: Optional[list] = None) -> torch.Tensor:
    chosen, score = router_choice(h @ w[f"{p}.router"].T, int(mlp["router"]["top"]), margins)
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        rows, place = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += gated(h[rows], w, f"{p}.e{e}", score[rows, place])
    if mlp.get("shared"):
        out = out + gated(h, w, f"{p}.shared")
    return st(out)


# ---- rotary positions -------------------------------------------------------------------------------------------
def rotary_tables(rot: dict, positions: torch.Tensor):
    dims, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / dims)
    mult = 1.0
    sc = rot.get("scaling")
    if sc:
        factor, original = float(sc["factor"]), float(sc["original"])

        def place(t):
            return dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))

        lo = max(math.floor(place(float(sc["fast"]))), 0)
        hi = min(math.ceil(place(float(sc["slow"]))), dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        f = f / factor * ramp + f * (1.0 - ramp)
        mult = 0.1 * math.log(factor) + 1.0
    ang = positions.to(torch.float64)[:, None] * f[None, :]
    return torch.cos(ang) * mult, torch.sin(ang) * mult


def turn(x: torch.Tensor, positions: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """``x [T, heads, d]``: pairs (2i, 2i + 1) of the first ``dims`` features turn with the position."""
    if not rot or not int(rot.get("dims", 0)):
        return x
    dims = int(rot["dims"])
    cos, sin = rotary_tables(rot, positions)
    cos, sin = cos.to(x.dtype)[:, None, :], sin.to(x.dtype)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


# ---- softmax attention ------------------------------------------------------------------------------------------
def visible_keys(T: int, window: Optional[int]) -> torch.Tensor:
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen & (i - j < window) if window else seen


def sink_softmax(scores: torch.Tensor, seen: torch.Tensor, sink) -> torch.Tensor:
    """``e^s_j / (e^sink + sum e^s)`` over the visible keys of each row."""
    scores = scores.masked_fill(~seen, float("-inf"))
    sink = torch.as_tensor(sink, dtype=scores.dtype).expand(scores.shape[0], 1)
    return torch.softmax(torch.cat([scores, sink], dim=-1), dim=-1)[:, :-1]


def temperature(positions: torch.Tensor, qt: Optional[dict], dtype) -> torch.Tensor:
    if not qt:
        return torch.ones(positions.shape[0], dtype=dtype)
    return 1.0 + float(qt["coef"]) * torch.log(torch.div(positions + 1, int(qt["every"]), rounding_mode="floor").to(dtype) + 1.0)


def attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q = unit(lin(h, w[f"{p}.q"]), eps) * w[f"{p}.q.norm"] * temperature(pos, m.get("q_temp"), h.dtype)[:, None]
    k = unit(lin(h, w[f"{p}.k"]), eps) * w[f"{p}.k.norm"]
    q, k = st(q).view(T, H, d), st(k).view(T, G, d)
    v = lin(h, w[f"{p}.v"]).view(T, G, dv)
    gate = torch.sigmoid(lin(h, w[f"{p}.g"]))
    seen = visible_keys(T, None)
    outs = []
    for hd in range(H):
        g = hd // (H // G)
        pr = sink_softmax((q[:, hd] @ k[:, g].T) * float(m["scale"]), seen, 0.0)
        outs.append((pr @ v[:, g]) * gate[:, hd:hd + 1])
    return lin(st(torch.cat(outs, dim=-1)), w[f"{p}.o"])


def latent_attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, dr, dv, r = (int(m[n]) for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    pos = torch.arange(T)
    cq = st(unit(lin(h, w[f"{p}.dq"]), eps) * w[f"{p}.dq.norm"])
    q = lin(cq, w[f"{p}.uq"]).view(T, H, d + dr)
    low = lin(h, w[f"{p}.dkv"])
    c = st(unit(low[:, :r], eps) * w[f"{p}.dkv.norm"])
    kr = st(turn(low[:, None, r:], pos, m.get("rot")))[:, 0]
    qr = st(turn(q[..., d:], pos, m.get("rot")))
    k = lin(c, w[f"{p}.uk"]).view(T, H, d)
    v = lin(c, w[f"{p}.uv"]).view(T, H, dv)
    mask = m.get("mask")
    seen = visible_keys(T, int(mask["size"]) if mask else None)
    outs = []
    for hd in range(H):
        s = (q[:, hd, :d] @ k[:, hd].T + qr[:, hd] @ kr.T) * float(m["scale"])
        outs.append(sink_softmax(s, seen, w[f"{p}.sink"][hd]) @ v[:, hd])
    return lin(st(torch.cat(outs, dim=-1)), w[f"{p}.o"])


# ---- recurrence -----------------------------------------------------------------------------------------------
def lightning(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, k = (st(F.silu(lin(h, w[f"{p}.{n}"]))).view(T, H, d) for n in "qk")
    v = st(F.silu(lin(h, w[f"{p}.v"]))).view(T, H, dv)
    decay = torch.tensor([float(x) for x in m["decay"]], dtype=h.dtype)[:, None, None]
    S = torch.zeros(H, d, dv, dtype=h.dtype)
    o = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    o = unit(o.reshape(T, H * dv), eps) * w[f"{p}.norm"] * torch.sigmoid(lin(h, w[f"{p}.g"]))
    return lin(st(o), w[f"{p}.o"])


# ---- the model --------------------------------------------------------------------------------------------------
MIXERS = {"attention": attention, "latent_attention": latent_attention, "lightning": lightning}


def layer(x: torch.Tensor, spec: dict, w: Dict[str, torch.Tensor], p: str, eps: float, alpha: float,
          margins: Optional[list] = None) -> torch.Tensor:
    y = MIXERS[spec["type"]](st(x), spec["mixer"], w, f"{p}.mix", eps)
    x = unit(alpha * x + w[f"{p}.ls1"] * y, eps) * w[f"{p}.norm1"]
    if spec.get("mlp") is not None:
        y = moe_ff(st(x), spec["mlp"], w, f"{p}.mlp", margins)
        x = unit(alpha * x + w[f"{p}.ls2"] * y, eps) * w[f"{p}.norm2"]
    return x


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64, streams: Optional[list] = None,
            margins: Optional[list] = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence; ``streams`` (a list) collects the stream after every layer, ``margins`` (a list)
    one tensor ``[T]`` per routed feed-forward: by how much its choice of experts was decided."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][tokens]
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, spec, w, f"l{i}", eps, float(cfg["postln_alpha"]), margins)
        if streams is not None:
            streams.append(x.clone())
    logits = st(unit(x, eps) * w["final.norm"]) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return float(cap) * torch.tanh(logits / float(cap)) if cap else logits


def random_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """Weights by checkpoint name for any configuration of this design, as bfloat16-representable float32 values.  Queries are
    sharpened (large norm weights, large query matrices) so that a wrong key shows; routers are decisive."""
    gen = torch.Generator().manual_seed(seed)
    W = int(cfg["width"])
    out: Dict[str, torch.Tensor] = {}

    def put(name, t):
        out[name] = t.to(torch.bfloat16).to(torch.float32)

    def mat(name, rows, cols, gain=1.0):
        put(name, torch.randn(rows, cols, generator=gen) * (gain / math.sqrt(cols)))

    def vec(name, n=W, mean=1.0):
        put(name, mean + 0.2 * mean * torch.randn(n, generator=gen))

    def glu(p, ff):
        mat(f"{p}.gate", ff, W)
        mat(f"{p}.up", ff, W)
        mat(f"{p}.down", W, ff)

    put("embed", torch.randn(int(cfg["vocab"]), W, generator=gen))
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}", spec["mixer"]
        for n in (1, 2) if spec.get("mlp") is not None else (1,):
            vec(f"{p}.norm{n}")
            vec(f"{p}.ls{n}", mean=1.5)
        q = f"{p}.mix"
        H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        if spec["type"] == "attention":
            G = int(m["kv_heads"])
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * dv), ("g", H)):
                mat(f"{q}.{n}", rows, W)
            vec(f"{q}.q.norm", H * d, 1.5)
            vec(f"{q}.k.norm", G * d)
        elif spec["type"] == "latent_attention":
            dr, r, qr = int(m["rot_dim"]), int(m["kv_rank"]), int(m["q_rank"])
            mat(f"{q}.dq", qr, W)
            vec(f"{q}.dq.norm", qr)
            mat(f"{q}.uq", H * (d + dr), qr, 1.5)
            mat(f"{q}.dkv", r + dr, W)
            vec(f"{q}.dkv.norm", r)
            mat(f"{q}.uk", H * d, r)
            mat(f"{q}.uv", H * dv, r)
            put(f"{q}.sink", torch.randn(H, generator=gen))
        else:
            for n, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
                mat(f"{q}.{n}", rows, W)
            vec(f"{q}.norm", H * dv)
        mat(f"{q}.o", W, H * dv)
        mlp = spec.get("mlp")
        if mlp is not None:
            mat(f"{p}.mlp.router", int(mlp["router"]["experts"]), W, 4.0)
            for e in range(int(mlp["router"]["experts"])):
                glu(f"{p}.mlp.e{e}", int(mlp["expert"]["ff"]))
            if mlp.get("shared"):
                glu(f"{p}.mlp.shared", int(mlp["shared"]["ff"]))
    vec("final.norm")
    mat("head", int(cfg["vocab"]), W, 4.0)
    return out
