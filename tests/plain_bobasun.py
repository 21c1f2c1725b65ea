"""The Bobasun decoder written out plainly and slowly in PyTorch, one function per mechanism, for the tests.

It shares no code with the package: it reads a configuration as a plain dict (the keys of ``config.json``) and weights
as a dict of tensors by checkpoint name, and computes everything in the dtype it is given (float64 by default), one
whole sequence at a time, with no cache and no state carried from call to call.

Notation: ``X`` is the bundle of residual streams ``[s, T, width]``.

    embedding:  X_1 = ... = X_s = E[tok] * c
    layer:      for each sublayer (mixer, then feed-forward if there is one) with its numbers a [s], M [s, s], b [s]:
                  y = sublayer(norm(sum_i a_i X_i)) ;  X_t <- sum_i M[i, t] X_i + b_t y      (all t from the old X)
    norm:       (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * w
    mixer:      q, k, v = W h + bias ; q, k turned by their positions (features j and j + dims/2 a pair, frequencies
                base^(-2j/dims) / factor), then divided by their root mean square per head ;
                v <- (1 - lambda) v + lambda v_first in all value-mixing layers but the first of them ;
                p_j = exp(s_j) / (1 + sum exp(s_j)), s = scale q.k, causal, grouped heads ;
                each head's output times sigmoid(W_g h) of that head ; W_o + bias
    ff:         g = min(W_gate h + bias, L), u = clamp(W_up h + bias, -L, L) ; W_down (g sigmoid(1.702 g) (u + 1)) + bias
    output:     logits = W_head norm(sum_i X_i)
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

SWISH_SLOPE = 1.702

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


def lin(x: torch.Tensor, w: torch.Tensor, b: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = x @ w.T
    return st(y if b is None else y + b)


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w


def unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


# ---- streams ----------------------------------------------------------------------------------------------------
def read_streams(X: torch.Tensor, a: torch.Tensor) -> torch.Tensor:
    """``X [s, T, w]``, ``a [s]`` -> ``[T, w]``."""
    out = torch.zeros_like(X[0])
    for i in range(X.shape[0]):
        out = out + a[i] * X[i]
    return out


def write_streams(X: torch.Tensor, y: torch.Tensor, M: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """``M[from, to]``; every new stream is made from the old ones."""
    new = []
    for t in range(X.shape[0]):
        x = b[t] * y
        for i in range(X.shape[0]):
            x = x + M[i, t] * X[i]
        new.append(x)
    return torch.stack(new)


# ---- attention --------------------------------------------------------------------------------------------------
def rotate(x: torch.Tensor, positions: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """``x [T, heads, d]``: features j and j + dims/2 (j < dims/2) turn with the position; the rest stays."""
    if not rot or not int(rot.get("dims", 0)):
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    out = x.clone()
    for j in range(dims // 2):
        ang = positions.to(torch.float64) * (base ** (-2.0 * j / dims) / factor)
        c, s = torch.cos(ang).to(x.dtype)[:, None], torch.sin(ang).to(x.dtype)[:, None]
        u, v = x[..., j], x[..., j + dims // 2]
        out[..., j] = u * c - v * s
        out[..., j + dims // 2] = v * c + u * s
    return out


def sink_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """``q [T, H, d]``, ``k [T, G, d]``, ``v [T, G, dv]`` -> ``[T, H, dv]``: causal, one added to the denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    hidden = torch.ones(T, T).triu(1).bool()
    outs = []
    for hd in range(H):
        g = hd // (H // G)
        s = ((q[:, hd] @ k[:, g].T) * scale).masked_fill(hidden, float("-inf"))
        top = s.max(dim=-1, keepdim=True).values.clamp(min=0.0)       # (the sink's own score is 0)
        e = torch.exp(s - top)
        p = e / (torch.exp(-top) + e.sum(-1, keepdim=True))
        outs.append(p @ v[:, g])
    return torch.stack(outs, dim=1)


def mix_values(v: torch.Tensor, first: torch.Tensor, lam: torch.Tensor) -> torch.Tensor:
    return (1 - lam) * v + lam * first


def attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float, values: dict) -> torch.Tensor:
    """``values``: what the layers of one forward pass share; ``values["first"]`` is set by the first value-mixing layer."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q = st(unit(rotate(lin(h, w[f"{p}.q"], w[f"{p}.q.b"]).view(T, H, d), pos, m.get("rot")), eps))
    k = st(unit(rotate(lin(h, w[f"{p}.k"], w[f"{p}.k.b"]).view(T, G, d), pos, m.get("rot")), eps))
    v = lin(h, w[f"{p}.v"], w[f"{p}.v.b"]).view(T, G, dv)
    if m.get("v_mix"):
        if "first" in values:
            v = st(mix_values(v, values["first"], w[f"{p}.vmix"]))
        else:
            values["first"] = v
    o = st(sink_attention(q, k, v, float(m["scale"])))
    gate = torch.sigmoid(lin(h, w[f"{p}.g"]))
    o = st(o * gate[:, :, None])
    return lin(o.reshape(T, H * dv), w[f"{p}.o"], w[f"{p}.o.b"])


# ---- feed-forward ---------------------------------------------------------------------------------------------
def clamped_glu(g: torch.Tensor, u: torch.Tensor, limit: float) -> torch.Tensor:
    g = torch.clamp(g, max=limit)
    u = torch.clamp(u, min=-limit, max=limit)
    return g * torch.sigmoid(SWISH_SLOPE * g) * (u + 1)


def feed_forward(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    g = lin(h, w[f"{p}.gate"], w[f"{p}.gate.b"])
    u = lin(h, w[f"{p}.up"], w[f"{p}.up.b"])
    return lin(st(clamped_glu(g, u, float(mlp["limit"]))), w[f"{p}.down"], w[f"{p}.down.b"])


# ---- the model --------------------------------------------------------------------------------------------------
def layer(X: torch.Tensor, entry: dict, w: Dict[str, torch.Tensor], p: str, eps: float, values: dict) -> torch.Tensor:
    steps = [("1", lambda h: attention(h, entry["mixer"], w, f"{p}.mix", eps, values))]
    if entry.get("mlp") is not None:
        steps.append(("2", lambda h: feed_forward(h, entry["mlp"], w, f"{p}.mlp")))
    for q, sublayer in steps:
        u = read_streams(X, w[f"{p}.hc{q}.in"])
        y = sublayer(st(layer_norm(u, w[f"{p}.norm{q}"], eps)))
        X = write_streams(X, y, w[f"{p}.hc{q}.mix"], w[f"{p}.hc{q}.out"])
    return X


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one whole sequence; ``layers_out`` (a list) gets the streams' sum after every layer."""
    w = {name: t.to(dtype) for name, t in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    X = torch.stack([x] * int(cfg.get("streams", 1)))
    values: dict = {}
    for i, entry in enumerate(cfg["layers"]):
        X = layer(X, entry, w, f"l{i}", eps, values)
        if layers_out is not None:
            layers_out.append(X.sum(0))
    h = st(layer_norm(X.sum(0), w["final.norm"], eps))
    return h @ w["head"].T


def greedy(cfg: dict, weights: Dict[str, torch.Tensor], prompt: List[int], n: int, dtype=torch.float64) -> List[int]:
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(forward(cfg, weights, tokens, dtype)[-1].argmax()))
    return tokens[len(prompt):]


def random_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """Random weights by checkpoint name, rounded to bfloat16: biases and mixing numbers large enough to matter, stream mixes
    that are far from the identity (but not growing), a different set of numbers for every sublayer."""
    gen = torch.Generator().manual_seed(seed)
    out: Dict[str, torch.Tensor] = {}

    def put(name, t):
        out[name] = t.to(torch.bfloat16).to(torch.float32)

    def mat(name, *shape, s):
        put(name, torch.randn(*shape, generator=gen) * s)

    def norm(name):
        put(name, 1.0 + 0.2 * torch.randn(W, generator=gen))

    V, W, S = int(cfg["vocab"]), int(cfg["width"]), int(cfg.get("streams", 1))
    mat("embed", V, W, s=1.0)
    mat("head", V, W, s=1.0 / math.sqrt(W))
    norm("final.norm")
    s_in = 1.0 / math.sqrt(W)
    for i, entry in enumerate(cfg["layers"]):
        p, m = f"l{i}", entry["mixer"]
        H, G, d, dv = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        for q in ("1", "2"):
            if q == "2" and entry.get("mlp") is None:
                continue
            norm(f"{p}.norm{q}")
            mat(f"{p}.hc{q}.in", S, s=1.0)
            mat(f"{p}.hc{q}.out", S, s=1.0)
            put(f"{p}.hc{q}.mix", 0.6 * torch.eye(S) + 0.5 / math.sqrt(S) * torch.randn(S, S, generator=gen))
        for name, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
            mat(f"{p}.mix.{name}", rows, W, s=s_in)
            mat(f"{p}.mix.{name}.b", rows, s=0.5)
        if m.get("v_mix"):
            put(f"{p}.mix.vmix", torch.rand((), generator=gen) * 0.8 + 0.1)
        mat(f"{p}.mix.g", H, W, s=2.0 * s_in)
        mat(f"{p}.mix.o", W, H * dv, s=1.0 / math.sqrt(H * dv))
        mat(f"{p}.mix.o.b", W, s=0.3)
        mlp = entry.get("mlp")
        if mlp is not None:
            ff = int(mlp["ff"])
            for name in ("gate", "up"):
                mat(f"{p}.mlp.{name}", ff, W, s=s_in)
                mat(f"{p}.mlp.{name}.b", ff, s=0.5)
            mat(f"{p}.mlp.down", W, ff, s=1.0 / math.sqrt(ff))
            mat(f"{p}.mlp.down.b", W, s=0.3)
    return out
