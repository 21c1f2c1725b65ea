"""The Burinex decoder as a plan of parts.

Every block is a ``norm_of_sum`` arrangement (``parts/block.py``): the stream is what the norm returns, ``x <- norm1(alpha x + ls1 *
mixer(x))``, then ``x <- norm2(alpha x + ls2 * ff(x))``, with one ``alpha`` for the model and a factor per feature on every
sublayer's output.  Layer by layer ``config.json`` chooses the mixer

* ``attention``: grouped-query softmax attention without positions, one RMS norm over all query heads and one over all key
  heads, a temperature on the queries that grows with the position, one added to the softmax's denominator, a sigmoid gate per
  head (``parts/attention.py``);
* ``latent_attention``: keys and values expanded from a cached low-rank row, queries through a latent of their own, a rotated
  part beside the keys (interleaved pairs, YaRN-scaled), a sliding window, a learned sink per head (``parts/latent_attention.py``);
* ``lightning``: a linear recurrence with a constant decay per head (``parts/lightning.py``);

and the feed-forward: none, or routed experts with sigmoid scores whose weights stand on the experts' inputs, with a shared
expert (``parts/moe.py``).  Final RMS norm, an output head of its own, logits capped by a tanh.

Tensor names: ``embed``, ``final.norm``, ``head``; layer i: ``l<i>.norm1, ls1, norm2, ls2``; ``l<i>.mix.{q,k,v,q.norm,k.norm,g,o}``
(attention), ``l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,sink,o}`` (latent) or ``l<i>.mix.{q,k,v,g,norm,o}`` (lightning);
``l<i>.mlp.router``, ``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.shared.{gate,up,down}``.
"""
from __future__ import annotations

from ..config.burinex import BurinexConfig
from ..config.registry import register_architecture
from ..parts.spec import BlockSpec, ModelPlan, PartSpec, RunStep


def burinex_plan(cfg: BurinexConfig) -> ModelPlan:
    h, eps = cfg.width, cfg.norm_eps
    norm = lambda name: PartSpec("rmsnorm", {"dim": h, "eps": eps}, {"weight": name})
    scale = lambda name: PartSpec("feature_scale", {"dim": h}, {"weight": name})
    positions = {}

    def position(spec: PartSpec) -> str:
        """One position encoding per distinct set of constants, shared by the layers that use it."""
        key = repr(sorted((k, repr(v)) for k, v in spec.params.items()))
        for name, have in positions.items():
            if repr(sorted((k, repr(v)) for k, v in have.params.items())) == key:
                return name
        name = f"rot{len(positions)}"
        positions[name] = spec
        return name

    def mixer(layer, q: str) -> PartSpec:
        m = layer.mixer
        names = lambda *ns: {n: f"{q}.{t}" for n, t in ns}
        if layer.type == "attention":
            temp = None if m.q_temp is None else {"coef": m.q_temp.coef, "every": m.q_temp.every}
            return PartSpec(
                "attention",
                {"hidden": h, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim, "qk_norm": "row",
                 "eps": eps, "scale": m.scale, "window": None, "position": None, "sink": True, "output_gate": "sigmoid_head",
                 "query_temperature": temp},
                names(("q_proj", "q"), ("k_proj", "k"), ("v_proj", "v"), ("q_norm", "q.norm"), ("k_norm", "k.norm"), ("g_proj", "g"),
                      ("o_proj", "o")))
        if layer.type == "latent_attention":
            pos = None
            if m.rot is not None and m.rot.dims > 0:
                sc = m.rot.scaling
                scaling = None if sc is None else {"factor": sc.factor, "original": sc.original, "fast": sc.fast, "slow": sc.slow}
                pos = position(PartSpec("rope", {"rotary_dim": m.rot.dims, "theta": m.rot.base, "style": "interleaved",
                                                 "scaling": scaling, "max_positions": cfg.max_positions, "exact": True}))
            return PartSpec(
                "latent_attention",
                {"hidden": h, "n_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_head_dim": m.vdim, "kv_rank": m.kv_rank,
                 "q_rank": m.q_rank, "scale": m.scale, "eps": eps, "gate": "none", "position": pos, "window": m.window, "sink": True},
                names(("dq_proj", "dq"), ("dq_norm", "dq.norm"), ("uq_proj", "uq"), ("dkv_proj", "dkv"), ("dkv_norm", "dkv.norm"),
                      ("uk_proj", "uk"), ("uv_proj", "uv"), ("sink", "sink"), ("o_proj", "o")))
        return PartSpec(
            "lightning",
            {"hidden": h, "n_heads": m.heads, "head_dim": m.dim, "v_head_dim": m.vdim, "decay": m.decay, "eps": eps},
            names(("q_proj", "q"), ("k_proj", "k"), ("v_proj", "v"), ("g_proj", "g"), ("norm", "norm"), ("o_proj", "o")))

    blocks = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}"
        parts = {"mixer": ("mixer", mixer(layer, f"{p}.mix")), "mixer_norm": ("norm", norm(f"{p}.norm1")),
                 "mixer_scale": ("stream", scale(f"{p}.ls1"))}
        f = layer.mlp
        if f is not None:
            q = f"{p}.mlp"
            weights = {"router": f"{q}.router"}
            for e in [f"e{j}" for j in range(f.experts)] + (["shared"] if f.shared_ff else []):
                weights.update({f"{e}.{s}": f"{q}.{e}.{s}" for s in ("gate", "up", "down")})
            parts["ffn"] = ("feed_forward", PartSpec(
                "routed_experts",
                {"hidden": h, "n_experts": f.experts, "n_identity": 0, "top": f.top, "intermediate": f.ff, "activation": "silu",
                 "choice": "sigmoid_groups", "weight_on": "input",
                 "shared": {"intermediate": f.shared_ff} if f.shared_ff else None}, weights))
            parts["ffn_norm"] = ("norm", norm(f"{p}.norm2"))
            parts["ffn_scale"] = ("stream", scale(f"{p}.ls2"))
        blocks.append(BlockSpec("norm_of_sum", parts, name=f"layer {i}", params={"alpha": cfg.postln_alpha}))
    # a layer without a feed-forward may still carry what stands around one in its file
    ignored = tuple(f"l{i}.{n}" for i, layer in enumerate(cfg.layers) if layer.mlp is None for n in ("norm2", "ls2"))
    return ModelPlan(
        hidden_size=h,
        vocab_size=cfg.vocab,
        max_positions=cfg.max_positions,
        embedding=PartSpec("token_embedding", {"vocab": cfg.vocab, "hidden": h}, {"weight": "embed"}),
        blocks=tuple(blocks),
        order=tuple(RunStep(block=i) for i in range(len(blocks))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab": cfg.vocab, "hidden": h, "softcap": cfg.logit_softcap}, {"weight": "head"}),
        positions=positions,
        ignored=ignored,
    )


register_architecture("Burinex", BurinexConfig, burinex_plan, replace=True)
