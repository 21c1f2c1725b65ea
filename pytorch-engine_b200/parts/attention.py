"""Grouped-query softmax attention over the paged cache, with optional per-head q/k RMSNorm,
optional rotary position encoding and an optional sliding window.

Order of operations (pygguf_engine/model.py:462-496): fused q|k|v projection, head split,
q/k-norm over head_dim (before RoPE, not on v), RoPE at position = cached length + row, append of
k, v to the cache, attention with scale ``1/sqrt(head_dim)`` unless the plan gives another
(pygguf_engine/model.py:281-284), merge heads, output projection.
"""
from __future__ import annotations

import math
from typing import Dict, Optional

import torch

from ..kernels import ops
from .linear import fuse_rows
from .registry import register
from .spec import CacheRequest, WeightDecl

# keys per partial result in decode: a property of the sequence, never of the batch (measured on the
# tensor-core kernels: 128 / 256 / 512 keys give 4,438 / 5,757 / 6,298 tokens/s at batch 64)
SPLIT_KEYS = 512


@register("mixer", "attention")
class GQAttention:
    """params: ``hidden``, ``n_heads``, ``n_kv_heads``, ``head_dim``, ``qk_norm`` (bool), ``eps``,
    ``scale`` (None: 1/sqrt(head_dim)), ``window`` (None: all keys), ``position`` (name of a position
    encoding of the plan, or None).  weights: ``q_proj, k_proj, v_proj, o_proj`` and, with qk_norm,
    ``q_norm, k_norm``.

    Further params, all optional: ``v_head_dim`` (values and head outputs of a size of their own), ``sink`` (true:
    one is added to the softmax's denominator, a key of score 0 that carries no value), ``v_norm`` ("unit": each
    head's value is divided by its root mean square, eps inside the root, no weight; it is cached so),
    ``value_position`` (name of a rotary encoding of the plan over the value's features: the value of position j is
    cached turned by j, and each head's output at position i is turned back by i before the output projection).
    A rotary ``position`` may use either layout of pairs.  ``bias`` (true: q, k and v have biases ``q_bias, k_bias, v_bias``,
    added in float32 before anything else), ``keep_first`` (with a ``window``: the first that many positions of a sequence stay
    visible to every later query, at their own positions), ``output_gate`` ("sigmoid": the joined heads are multiplied feature
    by feature with ``sigmoid(g_proj x)`` before the output projection; the gate's product rides in the q|k|v product).
    ``qk_norm`` may also be "row": q and k are each divided by the root mean square of all their heads together, with weights as
    long as the projections.  ``query_temperature`` ({"coef", "every"}): q at position p is multiplied by ``1 + coef *
    ln(floor((p + 1) / every) + 1)`` behind its norm (with ``qk_norm`` "row" or none).
    With any of these the mixer runs on the general kernels (``qkv_rotate_append``, ``attention_generic_ex``) unless a
    tensor-core kernel takes the case."""

    graph_safe = True  # launches only; nothing in forward() waits for the device

    @classmethod
    def weight_decls(cls, params) -> Dict[str, WeightDecl]:
        h, nh, nkv, d = (int(params[k]) for k in ("hidden", "n_heads", "n_kv_heads", "head_dim"))
        dv = int(params.get("v_head_dim") or d)
        decls = {
            "q_proj": WeightDecl((nh * d, h)),
            "k_proj": WeightDecl((nkv * d, h)),
            "v_proj": WeightDecl((nkv * dv, h)),
            "o_proj": WeightDecl((h, nh * dv)),
        }
        if params.get("qk_norm", False):
            row = params["qk_norm"] == "row"
            decls["q_norm"] = WeightDecl((nh * d if row else d,), "norm")
            decls["k_norm"] = WeightDecl((nkv * d if row else d,), "norm")
        if params.get("bias", False):
            decls.update({"q_bias": WeightDecl((nh * d,)), "k_bias": WeightDecl((nkv * d,)), "v_bias": WeightDecl((nkv * dv,))})
        if params.get("output_gate"):
            decls["g_proj"] = WeightDecl((nh if params["output_gate"] == "sigmoid_head" else nh * dv, h))
        if params.get("value_mix") == "mix":
            decls["v_lambda"] = WeightDecl((), "unit")
        if params.get("out_bias", False):
            decls["o_bias"] = WeightDecl((h,))
        return decls

    @classmethod
    def cache_request(cls, params) -> Optional[CacheRequest]:
        d = int(params["head_dim"])
        dv = int(params.get("v_head_dim") or d)
        return CacheRequest(kind="kv", kv_heads=int(params["n_kv_heads"]), head_dim=d, window=params.get("window"),
                            v_head_dim=None if dv == d else dv,
                            keep_first=int(params.get("keep_first") or 0) if params.get("window") else 0)

    def __init__(self, params, weights, runtime, positions=None) -> None:
        self.runtime = runtime
        self.hidden = int(params["hidden"])
        self.n_heads = int(params["n_heads"])
        self.n_kv_heads = int(params["n_kv_heads"])
        self.head_dim = int(params["head_dim"])
        if self.n_heads % self.n_kv_heads:
            raise ValueError("n_heads must be a multiple of n_kv_heads")
        self.v_dim = int(params.get("v_head_dim") or self.head_dim)
        if self.head_dim > 512 or self.v_dim > 512:
            raise ValueError(f"head_dim {self.head_dim} / v_head_dim {self.v_dim} is beyond what the attention kernels take (<= 512)")
        self.sink = bool(params.get("sink", False))
        self.v_norm = params.get("v_norm")
        if self.v_norm not in (None, "unit"):
            raise ValueError(f"v_norm {self.v_norm!r} is not built (None or 'unit')")
        self.eps = float(params.get("eps", 1e-6))
        scale = params.get("scale")
        self.scale = float(scale) if scale is not None else 1.0 / math.sqrt(self.head_dim)
        self.window = int(params["window"]) if params.get("window") else 0
        self.keep_first = int(params.get("keep_first") or 0) if self.window else 0
        if self.keep_first and (self.sink or params.get("value_position") is not None):
            raise ValueError("keep_first is not built together with a sink or turned values")
        self.output_gate = params.get("output_gate")
        if self.output_gate not in (None, "sigmoid", "sigmoid_head"):
            raise ValueError(f"output_gate {self.output_gate!r} is not built (None, 'sigmoid' or 'sigmoid_head')")
        self.qk_unit = bool(params.get("qk_unit", False))
        self.value_mix = params.get("value_mix")
        if self.value_mix not in (None, "keep", "mix"):
            raise ValueError(f"value_mix {self.value_mix!r} is not built (None, 'keep' or 'mix')")
        if self.value_mix == "mix" and self.v_norm:
            raise ValueError("value_mix is not built together with a norm on the values")
        # a single number, read once when the model is built
        self.v_lambda = float(weights["v_lambda"].to(torch.float32).reshape(-1)[0].item()) if self.value_mix == "mix" else 0.0
        self.out_bias = runtime.adopt(weights["o_bias"], torch.float32) if params.get("out_bias", False) else None
        self.out_bias_deferred = False
        self.bias = None
        if params.get("bias", False):
            self.bias = torch.cat([weights[n].to(device=runtime.device, dtype=torch.float32).reshape(-1)
                                   for n in ("q_bias", "k_bias", "v_bias")]).contiguous()
        fused = [weights["q_proj"], weights["k_proj"], weights["v_proj"]]
        if self.output_gate:
            fused.append(weights["g_proj"])       # q | k | v | gate: one product over the mixer's input
        if self.output_gate == "sigmoid_head":    # rows of the product stay 16-byte aligned
            rows = sum(t.shape[0] for t in fused)
            if rows % 8:
                fused.append(torch.zeros((8 - rows % 8, self.hidden), dtype=fused[0].dtype, device=fused[0].device))
        self.qkv = fuse_rows(runtime, fused)
        self.o_proj = runtime.adopt(weights["o_proj"])
        self.q_norm = self.k_norm = None
        if params.get("qk_norm", False):
            self.q_norm = runtime.adopt(weights["q_norm"], torch.float32)
            self.k_norm = runtime.adopt(weights["k_norm"], torch.float32)
        self.position = None
        self.fused_position = False
        name = params.get("position")
        if name is not None:
            self.position = (positions or {})[name]
            # a rotary encoding with tables is fused into the q/k-norm + append kernel; any other one is
            # applied by its own ``apply(q, k, positions)`` between that kernel's norm and its append
            self.fused_position = bool(getattr(self.position, "fusable_rotary", False))
            if not self.fused_position and not hasattr(self.position, "apply"):
                raise ValueError(f"position encoding {name!r} offers neither tables() nor apply(q, k, positions)")
        # one norm over all heads, a temperature on the queries: the append is the kernel that takes a token's whole row
        qk_norm = params.get("qk_norm", False)
        qt = params.get("query_temperature")
        self.temperature = None if not qt else (float(qt["coef"]), int(qt["every"]))
        if self.temperature is not None and self.temperature[1] <= 0:
            raise ValueError(f"query_temperature: 'every' must be positive, got {self.temperature[1]}")
        self.row_norm = qk_norm == "row" or self.temperature is not None
        if self.row_norm and ((qk_norm and qk_norm != "row") or self.bias is not None or self.qk_unit or self.value_mix
                              or self.v_norm or params.get("value_position") is not None):
            raise ValueError("a norm over all heads or a query temperature is not built together with a norm per head, biases, unit "
                             "queries, or normed, mixed or turned values")
        self.value_position = None
        vname = params.get("value_position")
        if vname is not None:
            self.value_position = (positions or {})[vname]
            if not getattr(self.value_position, "fusable_rotary", False):
                raise ValueError(f"value_position {vname!r} must be a rotary encoding with tables()")
            if self.value_position.tables()[2] > self.v_dim:
                raise ValueError(f"value_position {vname!r} rotates more features than a value has ({self.v_dim})")
        interleaved = self.fused_position and getattr(self.position, "interleaved", False)
        # what the kernels of the plain softmax attention do not do
        self.general = bool(self.sink or self.v_norm or self.value_position is not None or self.v_dim != self.head_dim
                            or interleaved or self.bias is not None or self.keep_first or self.output_gate or self.qk_unit
                            or self.value_mix or self.out_bias is not None or self.row_norm)
        if self.general and self.position is not None and not self.fused_position:
            raise ValueError("the general attention path takes a rotary position encoding with tables(), or none")
        self.qkv_dim = (self.n_heads + self.n_kv_heads) * self.head_dim + self.n_kv_heads * self.v_dim
        self.gate_col = self.qkv_dim               # the gate's columns follow q | k | v in the fused product
        if self.output_gate:
            self.qkv_dim = int(self.qkv.shape[0])
        # tensor-core kernels where they take the shape (bfloat16, head size 64 or 128, group <= 16);
        # the generic float32-arithmetic kernels otherwise
        # (with a sink or turned values too, if keys and values have one size and the values turn in interleaved pairs
        # over the whole head: these kernels take both in their epilogues)
        vp = self.value_position
        fast_ok = self.v_dim == self.head_dim and (vp is None or (getattr(vp, "interleaved", False)
                                                                  and vp.tables()[2] == self.v_dim))
        self.use_mma = (fast_ok and runtime.is_cuda
                        and ops.attention_mma_supported(runtime.dtype, self.head_dim, self.n_heads, self.n_kv_heads))
        # prefill on tcgen05 where that kernel takes the shape (bfloat16, head size 128, groups up to 32)
        self.use_umma_prefill = (fast_ok and runtime.is_cuda and not self.keep_first
                                 and ops.attention_umma_supported(runtime.dtype, self.head_dim, self.n_heads, self.n_kv_heads))
        # sizes that run in padded tiles, and a gate per head (no turned values)
        if self.general and vp is None and runtime.is_cuda:
            dims = (runtime.dtype, self.head_dim, self.v_dim, self.n_heads, self.n_kv_heads)
            self.use_mma = ops.attention_mma_dims_supported(*dims)
            self.use_umma_prefill = not self.keep_first and ops.attention_umma_dims_supported(*dims)
        self.generic_attention = bool(getattr(runtime, "generic_attention", False))   # comparisons: the general kernels only

    def forward(self, x: torch.Tensor, ctx, view, writes_cache: bool = True) -> torch.Tensor:
        rt = self.runtime
        n = x.shape[0]
        qkv = ctx.buffer("attn.qkv", (n, self.qkv_dim), rt.dtype)
        where = (ctx.token_seq, ctx.token_pos, ctx.seq_slot, ctx.seq_qstart, view.page_table, view.num_pages,
                 view.k_pages, view.v_pages)
        if self.general:
            if self.fuses_general_into_product(x, rt):
                # many rows: biases, unit norm, rotation, value mixing and the append ride in the product's epilogue
                cos = sin = None
                rotary_dim = 0
                if self.position is not None:
                    cos, sin, rotary_dim = self.position.tables()
                ops.gemm_umma2_qkv_rope(x, self.qkv, qkv, self.n_heads, self.n_kv_heads, self.head_dim, self.q_norm, self.k_norm,
                                        self.eps, cos, sin, rotary_dim, *where, writes_cache, rt.status, self.bias,
                                        **self.value_options(n, ctx))
            else:
                rt.linear(x, self.qkv, out=qkv)
                self.rotate_append_general(qkv, n, ctx, view, writes_cache)
            out = ctx.buffer("attn.out", (n, self.n_heads * self.v_dim), rt.dtype)
            self.attend_general(qkv, out, ctx, view)
            if self.output_gate == "sigmoid" or (self.output_gate and not self.gate_in_kernel(ctx)):
                gated = ctx.buffer("attn.gated", (n, self.n_heads * self.v_dim), rt.dtype)
                ops.sigmoid_gate(out.view(n, self.n_heads, self.v_dim).transpose(0, 1), self.gate_columns(qkv), gated)
                out = gated
            delta = ctx.buffer("attn.delta", (n, self.hidden), rt.dtype)
            rt.linear(out, self.o_proj, out=delta)
            if self.out_bias is not None and not self.out_bias_deferred:
                delta.add_(self.out_bias)
            return delta
        if self.fuses_rope_into_product(x, rt):
            # many rows: q/k-norm, rotation and the cache append ride in the epilogue of the q|k|v product (its
            # 256-column tiles are two whole heads), so q|k|v is never written and read again in between
            cos = sin = None
            rotary_dim = 0
            if self.position is not None:
                cos, sin, rotary_dim = self.position.tables()
            ops.gemm_umma2_qkv_rope(x, self.qkv, qkv, self.n_heads, self.n_kv_heads, self.head_dim, self.q_norm, self.k_norm,
                                    self.eps, cos, sin, rotary_dim, *where, writes_cache, rt.status)
        else:
            rt.linear(x, self.qkv, out=qkv)
            self.norm_rotate_append(qkv, n, ctx, view, writes_cache)
        out = ctx.buffer("attn.out", (n, self.n_heads * self.head_dim), rt.dtype)
        self.attend(qkv, out, ctx, view)
        delta = ctx.buffer("attn.delta", (n, self.hidden), rt.dtype)
        rt.linear(out, self.o_proj, out=delta)
        return delta

    def defer_out_bias(self) -> Optional[torch.Tensor]:
        """For an arrangement that adds the output projection's bias itself: the bias (float32, or None), which ``forward`` then
        leaves out."""
        self.out_bias_deferred = True
        return self.out_bias

    # ---- the general path ---------------------------------------------------------------------------------
    def rotate_append_general(self, qkv: torch.Tensor, n: int, ctx, view, writes_cache: bool) -> None:
        """q/k-norm, rotation of q and k, the values' norm and rotation, and the append, in one kernel."""
        cos = sin = vcos = vsin = None
        rot = vrot = 0
        inter = vinter = False
        if self.position is not None:
            cos, sin, rot = self.position.tables()
            inter = bool(getattr(self.position, "interleaved", False))
        if self.value_position is not None:
            vcos, vsin, vrot = self.value_position.tables()
            vinter = bool(getattr(self.value_position, "interleaved", False))
        if self.row_norm:
            ops.qkv_row_norm_append(qkv, n, self.n_heads, self.n_kv_heads, self.head_dim, self.v_dim, self.q_norm, self.k_norm,
                                    self.eps, self.temperature, cos, sin, rot, inter, ctx.token_seq, ctx.token_pos, ctx.seq_slot,
                                    ctx.seq_qstart, view.page_table, view.num_pages, view.k_pages, view.v_pages, writes_cache,
                                    self.runtime.status)
            return
        ops.qkv_rotate_append(qkv, n, self.n_heads, self.n_kv_heads, self.head_dim, self.v_dim, self.q_norm, self.k_norm,
                              self.eps, cos, sin, rot, inter, self.v_norm == "unit", vcos, vsin, vrot, vinter,
                              ctx.token_seq, ctx.token_pos, ctx.seq_slot, ctx.seq_qstart, view.page_table, view.num_pages,
                              view.k_pages, view.v_pages, writes_cache, self.runtime.status, self.bias,
                              **self.value_options(n, ctx))

    def value_options(self, n: int, ctx) -> dict:
        kept = None
        if self.value_mix:
            kept = ctx.buffer("attn.kept_values", (n, self.n_kv_heads * self.v_dim), self.runtime.dtype)
        return dict(qk_unit=self.qk_unit, v_mix=kept if self.value_mix == "mix" else None, v_lambda=self.v_lambda,
                    v_keep=kept if self.value_mix == "keep" else None)

    def fuses_general_into_product(self, x: torch.Tensor, rt) -> bool:
        """``fuses_rope_into_product`` for the general path: values as large as keys, neither normed nor turned; split-half pairs;
        with unit q and k a rotation that leaves lengths as they are, and not a norm with a weight as well."""
        if self.v_dim != self.head_dim or self.v_norm or self.value_position is not None or self.row_norm:
            return False
        if self.position is not None and getattr(self.position, "interleaved", False):
            return False
        if self.qk_unit and (self.q_norm is not None or (self.position is not None and not getattr(self.position, "keeps_lengths", False))):
            return False
        return self.fuses_rope_into_product(x, rt)

    def gate_columns(self, qkv: torch.Tensor) -> torch.Tensor:
        width = self.n_heads if self.output_gate == "sigmoid_head" else self.n_heads * self.v_dim
        return qkv[:, self.gate_col:self.gate_col + width]

    def gate_in_kernel(self, ctx) -> bool:
        """Whether the step's attention kernel multiplies the heads' gates in (the general kernels leave it to one behind)."""
        if self.output_gate != "sigmoid_head" or self.generic_attention:
            return False
        return self.use_mma or (self.use_umma_prefill and not ctx.decode)

    def attend_general(self, q: torch.Tensor, out: torch.Tensor, ctx, view) -> None:
        vcos = vsin = None
        vrot = 0
        vinter = False
        if self.value_position is not None:
            vcos, vsin, vrot = self.value_position.tables()
            vinter = bool(getattr(self.value_position, "interleaved", False))
        where = (ctx.seq_qstart, ctx.seq_past, ctx.seq_slot, view.page_table, view.num_pages, view.k_pages, view.v_pages)
        extra = dict(sink=self.sink, out_cos=vcos, out_sin=vsin)
        gate = self.gate_columns(q) if self.gate_in_kernel(ctx) else None
        if self.use_umma_prefill and not ctx.decode and not self.generic_attention:
            ops.attention_umma_prefill(q, out, ctx.n_seqs, ctx.max_q, self.n_heads, self.n_kv_heads, self.head_dim, self.scale,
                                       self.window, *where, self.runtime.status, v_dim=self.v_dim, gate=gate, **extra)
            return
        if self.use_mma and not self.generic_attention:
            scratch = None
            split_keys, max_splits, floor = SPLIT_KEYS, 0, 0
            if ctx.decode:
                split_keys, max_splits, floor = ops.attention_mma_decode_ranges(
                    q.device, self.head_dim, ctx.n_seqs, self.n_kv_heads, ctx.max_kv_len, SPLIT_KEYS, v_dim=self.v_dim)
                scratch = ctx.buffer(
                    "attn.scratch",
                    (ops.attention_generic_scratch_floats(ctx.n_seqs, self.n_heads, self.v_dim, max_splits),), torch.float32)
            if self.value_position is None:
                ops.attention_mma_gated(ctx.decode, q, out, ctx.n_seqs, ctx.max_q, self.n_heads, self.n_kv_heads, self.head_dim,
                                        self.v_dim, self.scale, self.window, *where, scratch, split_keys, max_splits,
                                        self.runtime.status, min_range_keys=floor, sink=self.sink, gate=gate,
                                        keep_first=self.keep_first)
                return
            ops.attention_mma(ctx.decode, q, out, ctx.n_seqs, ctx.max_q, self.n_heads, self.n_kv_heads, self.head_dim,
                              self.scale, self.window, *where, scratch, split_keys, max_splits, self.runtime.status,
                              min_range_keys=floor, **extra)
            return
        scratch = None
        max_splits = 0
        if ctx.decode:
            max_splits = ctx.max_splits(SPLIT_KEYS)
            scratch = ctx.buffer(
                "attn.scratch",
                (ops.attention_generic_scratch_floats(ctx.n_seqs, self.n_heads, self.v_dim, max_splits),), torch.float32)
        if self.keep_first:
            ops.attention_generic_masked(
                ctx.decode, q, out, ctx.n_seqs, ctx.max_q, self.n_heads, self.n_kv_heads, self.head_dim, self.v_dim,
                self.scale, ctx.seq_qstart, ctx.seq_past, ctx.seq_slot, view.page_table, view.num_pages, view.k_pages,
                view.v_pages, scratch, SPLIT_KEYS, max_splits, self.runtime.status, window=self.window,
                keep_first=self.keep_first)
            return
        ops.attention_generic_ex(
            ctx.decode, q, out, ctx.n_seqs, ctx.max_q, self.n_heads, self.n_kv_heads, self.head_dim, self.v_dim,
            self.scale, self.window, self.sink, vcos, vsin, vrot, vinter, ctx.seq_qstart, ctx.seq_past, ctx.seq_slot,
            view.page_table, view.num_pages, view.k_pages, view.v_pages, scratch, SPLIT_KEYS, max_splits,
            self.runtime.status)

    def fuses_rope_into_product(self, x: torch.Tensor, rt) -> bool:
        """Whether this step's q|k|v product takes norm, rotation and append into its epilogue: the many-row tcgen05
        pair kernel must be the one that runs (as ``Runtime.linear`` would decide), the position encoding one that
        it can apply (rotary tables over the whole head, or none), the head size 128."""
        if rt.gemm_backend is not None or not rt.fuse_qkv_rope or not rt.pair_gemm or not rt.takes_large_gemm(x, self.qkv):
            return False
        if self.position is not None and not self.fused_position:
            return False
        rotary_dim = self.position.tables()[2] if self.position is not None else 0
        return ops.gemm_umma2_qkv_rope_supported(x, self.qkv, self.n_heads, self.n_kv_heads, self.head_dim, rotary_dim)

    def norm_rotate_append(self, qkv: torch.Tensor, n: int, ctx, view, writes_cache: bool) -> None:
        """q/k-norm, position encoding and cache append on the projected rows, as kernels of their own."""
        rt = self.runtime
        where = (ctx.token_seq, ctx.token_pos, ctx.seq_slot, ctx.seq_qstart, view.page_table, view.num_pages,
                 view.k_pages, view.v_pages)
        shape = (qkv, n, self.n_heads, self.n_kv_heads, self.head_dim)
        if self.position is None or self.fused_position:
            cos = sin = None
            rotary_dim = 0
            if self.position is not None:
                cos, sin, rotary_dim = self.position.tables()
            ops.qk_norm_rope_append(*shape, self.q_norm, self.k_norm, self.eps, cos, sin, rotary_dim, *where,
                                    writes_cache, rt.status)
        else:
            # in the order of the fused kernel: q/k-norm in place, then the position encoding's own code on
            # q and k (views of the fused buffer, [N, heads, head_dim]), then the append of k and v
            if self.q_norm is not None:
                ops.qk_norm_rope_append(*shape, self.q_norm, self.k_norm, self.eps, None, None, 0, *where, False, rt.status)
            qd, kd = self.n_heads * self.head_dim, self.n_kv_heads * self.head_dim
            self.position.apply(qkv[:, :qd].view(n, self.n_heads, self.head_dim),
                                qkv[:, qd:qd + kd].view(n, self.n_kv_heads, self.head_dim), ctx.token_pos)
            if writes_cache:
                ops.qk_norm_rope_append(*shape, None, None, self.eps, None, None, 0, *where, True, rt.status)

    def attend(self, q: torch.Tensor, out: torch.Tensor, ctx, view) -> None:
        """Attention of the step's queries (the first ``n_heads*head_dim`` features of each row of
        ``q``) over the cache of their sequences."""
        if self.use_umma_prefill and not ctx.decode:
            ops.attention_umma_prefill(
                q, out, ctx.n_seqs, ctx.max_q, self.n_heads, self.n_kv_heads, self.head_dim, self.scale, self.window,
                ctx.seq_qstart, ctx.seq_past, ctx.seq_slot, view.page_table, view.num_pages, view.k_pages, view.v_pages,
                self.runtime.status)
            return
        scratch = None
        max_splits = 0
        split_keys = SPLIT_KEYS
        extra = {}
        if ctx.decode:
            if self.use_mma:
                split_keys, max_splits, floor = ops.attention_mma_decode_ranges(
                    q.device, self.head_dim, ctx.n_seqs, self.n_kv_heads, ctx.max_kv_len, SPLIT_KEYS)
                extra["min_range_keys"] = floor
            else:
                max_splits = ctx.max_splits(split_keys)
            scratch = ctx.buffer(
                "attn.scratch",
                (ops.attention_generic_scratch_floats(ctx.n_seqs, self.n_heads, self.head_dim, max_splits),),
                torch.float32)
        kernel = ops.attention_mma if self.use_mma else ops.attention_generic
        kernel(
            ctx.decode, q, out, ctx.n_seqs, ctx.max_q, self.n_heads, self.n_kv_heads, self.head_dim, self.scale,
            self.window, ctx.seq_qstart, ctx.seq_past, ctx.seq_slot, view.page_table, view.num_pages, view.k_pages,
            view.v_pages, scratch, split_keys, max_splits, self.runtime.status, **extra)
