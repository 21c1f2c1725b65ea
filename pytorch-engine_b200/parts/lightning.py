"""Lightning attention: a linear recurrence with one constant decay per head (the kernels: csrc/ssd.cu).

For a token with input ``h``, per head with key size ``d`` and value size ``dv``:

    q, k, v = silu(W_q h), silu(W_k h), silu(W_v h)
    S <- decay S + k v^T ;  o = S^T q                       S [d, dv], float32
    out = W_o (unit(all heads) * norm * sigmoid(W_g h))     one root mean square over the concatenated heads

What a sequence keeps between steps is of fixed size: every head's ``S``, float32 (a "state" entry of the cache, zero when a
slot is taken).  The recurrence, its inputs behind the projections, the norm and the gate are float32 in every run dtype.
"""
from __future__ import annotations

import math
from typing import Dict, Optional

import torch

from ..kernels import ops
from .linear import fuse_rows
from .registry import register
from .spec import CacheRequest, WeightDecl

# tokens per chunk when a prompt is cut into chunks that run side by side; steps whose longest sequence has at most two
# chunks walk each sequence in one go
CHUNK_TOKENS = 64


@register("mixer", "lightning")
class LightningMixer:
    """params: ``hidden``, ``n_heads``, ``head_dim``, ``v_head_dim``, ``decay`` (one number a head), ``eps`` (of the norm).
    weights: ``q_proj, k_proj [heads*d, hidden]``, ``v_proj, g_proj [heads*dv, hidden]``, ``norm [heads*dv]``, ``o_proj [hidden,
    heads*dv]``."""

    graph_safe = True  # launches only; nothing in forward() waits for the device

    @classmethod
    def sizes(cls, params):
        return tuple(int(params[k]) for k in ("hidden", "n_heads", "head_dim", "v_head_dim"))

    @classmethod
    def weight_decls(cls, params) -> Dict[str, WeightDecl]:
        h, nh, d, dv = cls.sizes(params)
        return {"q_proj": WeightDecl((nh * d, h)), "k_proj": WeightDecl((nh * d, h)), "v_proj": WeightDecl((nh * dv, h)),
                "g_proj": WeightDecl((nh * dv, h)), "norm": WeightDecl((nh * dv,), "norm"), "o_proj": WeightDecl((h, nh * dv))}

    @classmethod
    def cache_request(cls, params) -> Optional[CacheRequest]:
        _, nh, d, dv = cls.sizes(params)
        return CacheRequest(kind="state", state_shapes=(("S", (nh, d, dv), "float32"),))

    def __init__(self, params, weights, runtime) -> None:
        self.runtime = runtime
        self.hidden, self.n_heads, self.head_dim, self.v_dim = self.sizes(params)
        self.eps = float(params.get("eps", 1e-6))
        decay = [float(x) for x in params["decay"]]
        if len(decay) != self.n_heads or any(not 0.0 <= x <= 1.0 for x in decay):
            raise ValueError(f"a lightning mixer of {self.n_heads} heads needs as many decays in [0, 1], got {decay}")
        d, dv = self.head_dim, self.v_dim
        if dv > 1024 or (d > 128 and (d * dv + 64 * d + 32 * dv) * 4 > 200 * 1024):
            raise ValueError(f"a head of {d} x {dv} is beyond what the recurrence kernel keeps on chip")
        f32 = torch.float32
        self.decay = torch.tensor(decay, dtype=f32, device=runtime.device)
        self.log_decay = torch.tensor([math.log(x) if x > 0.0 else -math.inf for x in decay], dtype=f32, device=runtime.device)
        self.qkvg = fuse_rows(runtime, [weights[f"{n}_proj"] for n in "qkvg"])
        self.norm = runtime.adopt(weights["norm"], f32)
        self.o_proj = runtime.adopt(weights["o_proj"])

    def forward(self, x: torch.Tensor, ctx, view, writes_cache: bool = True) -> torch.Tensor:
        if not writes_cache:
            raise ValueError("a lightning mixer folds every token into its state; it cannot run without writing it")
        rt = self.runtime
        n, nh, d, dv = x.shape[0], self.n_heads, self.head_dim, self.v_dim
        qkv, inner = nh * (2 * d + dv), nh * dv
        wide = ctx.buffer("lightning.qkvg", (n, qkv + inner), rt.dtype)
        rt.linear(x, self.qkvg, out=wide)
        y = ctx.buffer("lightning.y", (n, inner), torch.float32)
        chunk, max_chunks, scratch = 0, 1, None
        if ctx.max_q > 2 * CHUNK_TOKENS:
            chunk = CHUNK_TOKENS
            max_chunks = -(-ctx.max_q // chunk)
            scratch = ctx.buffer("lightning.scratch", (ops.ssd_scratch_floats(ctx.n_seqs, nh, d, dv, max_chunks),), torch.float32)
        ops.lightning_recurrence(wide[:, :qkv], self.decay, self.log_decay, y, view.state("S"), ctx.seq_slot, ctx.seq_qstart,
                                 ctx.n_seqs, ctx.max_q, nh, d, dv, rt.status, chunk, max_chunks, scratch)
        normed = ctx.buffer("lightning.normed", (n, inner), rt.dtype)
        ops.gated_part_norm(y, wide[:, qkv:], self.norm, self.eps, normed, 1, gate_first=False)
        delta = ctx.buffer("lightning.delta", (n, self.hidden), rt.dtype)
        rt.linear(normed, self.o_proj, out=delta)
        return delta
