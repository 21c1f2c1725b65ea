"""The Bobasun decoder as a plan of parts.

The embedding's rows are multiplied by ``embedding.scale``.  Every block is a ``streams`` arrangement (``parts/block.py``):
``streams`` residual streams side by side, each sublayer reading a learned mix of them through a layer norm and writing its
output back into all of them.  The mixer is grouped-query softmax attention (``parts/attention.py``) with biases, split-half
rotary pairs on the first ``rot.dims`` features with linearly scaled frequencies, q and k of unit root mean square after the
rotation, one added to the softmax's denominator, values mixed with the values of the first ``v_mix`` layer, and a sigmoid gate
per head.  The feed-forward: none, or a clamped gated one with biases (``parts/swiglu.py``).  Final layer norm of the streams'
sum; an output head of its own.

Tensor names: ``embed``, ``final.norm``, ``head``; layer i: ``l<i>.norm1, norm2``; ``l<i>.mix.{q,k,v,o}`` each with ``.b``,
``l<i>.mix.{g,vmix}``; ``l<i>.mlp.{gate,up,down}`` each with ``.b``; ``l<i>.hc1.{in,mix,out}`` (mixer) and ``l<i>.hc2.{in,mix,out}``
(feed-forward).
"""
from __future__ import annotations

from ..config.bobasun import BobasunConfig
from ..config.registry import register_architecture
from ..parts.spec import BlockSpec, ModelPlan, PartSpec, RunStep

# the slope of the sigmoid in the feed-forward's gate
SWISH_SLOPE = 1.702


def bobasun_plan(cfg: BobasunConfig) -> ModelPlan:
    h, eps = cfg.width, cfg.norm_eps
    norm = lambda name: PartSpec("layer_norm", {"dim": h, "eps": eps}, {"weight": name})
    bundle = lambda p: PartSpec("stream_bundle", {"streams": cfg.streams}, {"read": f"{p}.in", "mix": f"{p}.mix", "write": f"{p}.out"})
    positions = {}
    blocks = []
    ignored = []
    mixed = False         # a layer with value mixing has come by
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}"
        m = layer.mixer
        q = f"{p}.mix"
        pos = None
        if m.rot_dims > 0:
            # one position encoding per distinct set of constants, shared by the layers that use it
            pos = f"rot_{m.rot_dims}_{m.rot_base!r}_{m.rot_factor!r}"
            positions[pos] = PartSpec("rope", {"rotary_dim": m.rot_dims, "theta": m.rot_base, "style": "neox",
                                               "scaling": {"factor": m.rot_factor}, "max_positions": cfg.max_positions, "exact": True})
        names = {f"{s}_proj": f"{q}.{s}" for s in ("q", "k", "v", "g", "o")}
        names.update({f"{s}_bias": f"{q}.{s}.b" for s in ("q", "k", "v", "o")})
        value_mix = None
        if m.v_mix:
            value_mix = "mix" if mixed else "keep"
            mixed = True
        if value_mix == "mix":
            names["v_lambda"] = f"{q}.vmix"
        else:
            ignored.append(f"{q}.vmix")      # a layer that mixes nothing in may still carry the number
        parts = {
            "mixer_norm": ("norm", norm(f"{p}.norm1")),
            "mixer": ("mixer", PartSpec(
                "attention",
                {"hidden": h, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim,
                 "qk_norm": False, "qk_unit": True, "eps": eps, "scale": m.scale, "window": None, "position": pos, "sink": True,
                 "bias": True, "out_bias": True, "output_gate": "sigmoid_head", "value_mix": value_mix}, names)),
            "mixer_streams": ("stream", bundle(f"{p}.hc1")),
        }
        mlp = layer.mlp
        if mlp is not None:
            q = f"{p}.mlp"
            names = {f"{s}_proj": f"{q}.{s}" for s in ("gate", "up", "down")}
            names.update({f"{s}_bias": f"{q}.{s}.b" for s in ("gate", "up", "down")})
            parts["ffn_norm"] = ("norm", norm(f"{p}.norm2"))
            parts["ffn"] = ("feed_forward", PartSpec(
                "swiglu", {"hidden": h, "intermediate": mlp.ff, "activation": "clamped_swish", "limit": mlp.limit,
                           "alpha": SWISH_SLOPE, "bias": True}, names))
            parts["ffn_streams"] = ("stream", bundle(f"{p}.hc2"))
        else:
            # a layer without a feed-forward may still carry what stands around one in its file
            ignored += [f"{p}.norm2"] + [f"{p}.hc2.{s}" for s in ("in", "mix", "out")]
        blocks.append(BlockSpec("streams", parts, name=f"layer {i}"))
    return ModelPlan(
        hidden_size=h,
        vocab_size=cfg.vocab,
        max_positions=cfg.max_positions,
        embedding=PartSpec("token_embedding", {"vocab": cfg.vocab, "hidden": h, "scale": cfg.embedding_scale}, {"weight": "embed"}),
        blocks=tuple(blocks),
        order=tuple(RunStep(block=i) for i in range(len(blocks))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab": cfg.vocab, "hidden": h}, {"weight": "head"}),
        positions=positions,
        ignored=tuple(ignored),
    )


register_architecture("Bobasun", BobasunConfig, bobasun_plan, replace=True)
