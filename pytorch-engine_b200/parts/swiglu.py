"""SwiGLU feed-forward: ``down(silu(gate(x)) * up(x))`` with gate|up as one product
(pygguf_engine/model.py:839-846, pygguf_engine/quant_kernels.py:1467-1472)."""
from __future__ import annotations

from typing import Dict

import torch

from ..kernels import ops
from .linear import fuse_rows
from .registry import register
from .spec import WeightDecl


@register("feed_forward", "swiglu")
class SwiGLU:
    """params: ``hidden``, ``intermediate``.  weights: ``gate_proj, up_proj [I, H]``, ``down_proj [H, I]``.

    Optional params: ``activation`` ("silu", the default; "relu": ``relu(gate) * up``; "clamped_swish": ``g' sigmoid(alpha
    g') (u' + 1)`` with ``g' = min(gate, limit)``, ``u' = clamp(up, -limit, limit)``), with ``limit`` and ``alpha``; ``bias``
    (true: all three projections have biases ``gate_bias, up_bias, down_bias``; an arrangement that adds the last one itself
    calls ``defer_out_bias``).  Activation and biases ride in the epilogues of the package's product kernels; behind a
    library product they are a kernel of their own."""

    graph_safe = True  # launches only; nothing in forward() waits for the device

    @classmethod
    def weight_decls(cls, params) -> Dict[str, WeightDecl]:
        h, i = int(params["hidden"]), int(params["intermediate"])
        decls = {"gate_proj": WeightDecl((i, h)), "up_proj": WeightDecl((i, h)), "down_proj": WeightDecl((h, i))}
        if params.get("bias", False):
            decls.update({"gate_bias": WeightDecl((i,)), "up_bias": WeightDecl((i,)), "down_bias": WeightDecl((h,))})
        return decls

    def __init__(self, params, weights, runtime) -> None:
        self.runtime = runtime
        self.hidden = int(params["hidden"])
        self.intermediate = int(params["intermediate"])
        self.activation = str(params.get("activation") or "silu")
        if self.activation not in ops.GLU_KINDS:
            raise ValueError(f"activation {self.activation!r} is not built ({', '.join(sorted(ops.GLU_KINDS))} are)")
        self.limit = float(params.get("limit") or 0.0)
        self.alpha = float(params.get("alpha") or 1.0)
        self.gate_up = fuse_rows(runtime, [weights["gate_proj"], weights["up_proj"]])
        self.down = runtime.adopt(weights["down_proj"])
        self.bias = self.out_bias = None
        self.out_bias_deferred = False
        if params.get("bias", False):
            self.bias = torch.cat([weights[n].to(device=runtime.device, dtype=torch.float32).reshape(-1)
                                   for n in ("gate_bias", "up_bias")]).contiguous()
            self.out_bias = runtime.adopt(weights["down_bias"], torch.float32)
        # the activation for the fused epilogues (None: SiLU without biases, their default)
        self.glu = None
        if self.activation != "silu" or self.bias is not None:
            self.glu = (self.activation, self.limit, self.alpha, self.bias)

    def defer_out_bias(self):
        """For an arrangement that adds the down projection's bias itself: the bias (float32, or None), which ``forward`` then
        leaves out."""
        self.out_bias_deferred = True
        return self.out_bias

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        rt = self.runtime
        n = x.shape[0]
        act = ctx.buffer("ffn.act", (n, self.intermediate), rt.dtype)
        if rt.takes_small_gemm(x, self.gate_up):
            # few rows: gate|up product with the activation in its epilogue
            ops.gemm_smallm(x, self.gate_up, act, pair_offset=self.intermediate, glu=self.glu)
        elif rt.takes_large_gemm(x, self.gate_up, self.intermediate):
            # tcgen05 product over [gate rows | matching up rows] tiles, gate applied on the way out of TMEM
            # many rows: a pair of SMs per tile where the kernel takes the shape (K a multiple of 64)
            pair = rt.pair_gemm and x.shape[0] >= rt.large_gemm_rows and ops.gemm_umma2_supported(x, self.gate_up, self.intermediate)
            (ops.gemm_umma2 if pair else ops.gemm_umma)(x, self.gate_up, act, rt.status, pair_offset=self.intermediate, glu=self.glu)
        else:
            gu = ctx.buffer("ffn.gate_up", (n, 2 * self.intermediate), rt.dtype)
            rt.linear(x, self.gate_up, out=gu)
            if self.glu is None:
                ops.silu_mul(gu, act)
            else:
                ops.glu_act(gu, act, self.activation, self.limit, self.alpha, self.bias)
        delta = ctx.buffer("ffn.delta", (n, self.hidden), rt.dtype)
        rt.linear(act, self.down, out=delta)
        if self.out_bias is not None and not self.out_bias_deferred:
            delta.add_(self.out_bias)
        return delta
