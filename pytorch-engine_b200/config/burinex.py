"""Typed configuration of the Burinex decoder, read from its own ``config.json`` keys.

    {"architecture": "Burinex", "vocab": V, "width": W, "norm": {"eps": e}, "postln_alpha": a, "logit_softcap": c,
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "q_temp": {"coef", "every"}},
                 "mlp": {"kind": "moe", "router": {"experts", "top"}, "expert": {"ff"}, "shared": {"ff"}}},
                {"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "mask": {"size"},
                           "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"}}}, "mlp": ...},
                {"type": "lightning", "mixer": {"heads", "dim", "vdim", "decay": [one a head]}, "mlp": null}, ...]}

Every size and constant is read from there, layer by layer; nothing is the same for two layers unless the file says so.
"""
from __future__ import annotations

import os
from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, ModelConfig, require_float, require_int
from .registry import register_preset_folder
from .vabelorn import Rotary, _obj, _rotary, _sub

# The file gives no longest sequence; position tables are made for what the engine is asked to hold, up to this.
MAX_POSITIONS = 1 << 17


@dataclass(frozen=True)
class QueryTemperature:
    coef: float
    every: int


@dataclass(frozen=True)
class RowNormAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: Optional[QueryTemperature]


@dataclass(frozen=True)
class WindowLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    window: Optional[int]
    rot: Optional[Rotary]


@dataclass(frozen=True)
class Lightning:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class RoutedFf:
    experts: int
    top: int
    ff: int
    shared_ff: int     # 0: no shared expert


@dataclass(frozen=True)
class BurinexLayer:
    type: str                       # "attention" | "latent_attention" | "lightning"
    mixer: Any                      # RowNormAttention | WindowLatent | Lightning
    mlp: Optional[RoutedFf]


def _mlp(d: Any, where: str) -> Optional[RoutedFf]:
    if d is None:
        return None
    d = _obj(d, where)
    kind = d.get("kind", "moe")
    if kind != "moe":
        raise ConfigError(f"config.json: {where}: 'kind' must be 'moe', got {kind!r}")
    rwhole, _ = _sub(_obj(d.get("router"), where + ".router"), where + ".router")
    experts, top = rwhole("experts"), rwhole("top")
    if top > experts:
        raise ConfigError(f"config.json: {where}.router: 'top' ({top}) exceeds 'experts' ({experts})")
    ewhole, _ = _sub(_obj(d.get("expert"), where + ".expert"), where + ".expert")
    shared = 0
    if d.get("shared"):
        swhole, _ = _sub(_obj(d["shared"], where + ".shared"), where + ".shared")
        shared = swhole("ff")
    return RoutedFf(experts=experts, top=top, ff=ewhole("ff"), shared_ff=shared)


def _mixer(kind: Any, m: Dict[str, Any], where: str):
    whole, num = _sub(m, where)
    if kind == "attention":
        heads, kv = whole("heads"), whole("kv_heads", default=m.get("heads"))
        if heads % kv:
            raise ConfigError(f"config.json: {where}: 'heads' ({heads}) must be a multiple of 'kv_heads' ({kv})")
        dim = whole("dim")
        temp = None
        if m.get("q_temp"):
            twhole, tnum = _sub(_obj(m["q_temp"], where + ".q_temp"), where + ".q_temp")
            temp = QueryTemperature(coef=tnum("coef", positive=False), every=twhole("every"))
        return RowNormAttention(heads=heads, kv_heads=kv, dim=dim, vdim=whole("vdim", default=dim), scale=num("scale"), q_temp=temp)
    if kind == "latent_attention":
        dim, rot_dim = whole("dim"), whole("rot_dim", minimum=0, default=0)
        rot = _rotary(m["rot"], where + ".rot", rot_dim) if m.get("rot") else None
        window = None
        if m.get("mask"):
            mwhole, _ = _sub(_obj(m["mask"], where + ".mask"), where + ".mask")
            window = mwhole("size")
        return WindowLatent(heads=whole("heads"), dim=dim, rot_dim=rot_dim, vdim=whole("vdim", default=dim), kv_rank=whole("kv_rank"),
                            q_rank=whole("q_rank"), scale=num("scale"), window=window, rot=rot)
    if kind == "lightning":
        heads, dim = whole("heads"), whole("dim")
        decay = m.get("decay")
        if not isinstance(decay, (list, tuple)) or len(decay) != heads or any(
                isinstance(x, bool) or not isinstance(x, (int, float)) or not 0.0 <= x <= 1.0 for x in decay):
            raise ConfigError(f"config.json: {where}: 'decay' must list one number in [0, 1] for each of the {heads} heads, got {decay!r}")
        return Lightning(heads=heads, dim=dim, vdim=whole("vdim", default=dim), decay=tuple(float(x) for x in decay))
    raise ConfigError(f"config.json: {where[:-len('.mixer')]}: 'type' must be 'attention', 'latent_attention' or 'lightning', got {kind!r}")


@dataclass(frozen=True)
class BurinexConfig(ModelConfig):
    vocab: int
    width: int
    layers: Tuple[BurinexLayer, ...]
    norm_eps: float
    postln_alpha: float = 1.0
    logit_softcap: float = 0.0      # 0: the logits are not capped
    eos_token_id: Tuple[int, ...] = ()
    bos_token_id: Optional[int] = None
    architecture: str = field(default="Burinex")

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "BurinexConfig":
        vocab, width = require_int(d, "vocab"), require_int(d, "width")
        _, nnum = _sub(_obj(d.get("norm"), "'norm'"), "'norm'")
        raw = d.get("layers")
        if not isinstance(raw, (list, tuple)) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw):
            where = f"layers[{i}]"
            entry = _obj(entry, where)
            kind = entry.get("type")
            mixer = _mixer(kind, _obj(entry.get("mixer"), where + ".mixer"), where + ".mixer")
            layers.append(BurinexLayer(type=kind, mixer=mixer, mlp=_mlp(entry.get("mlp"), where + ".mlp")))
        cap = 0.0 if d.get("logit_softcap") is None else require_float(d, "logit_softcap")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else (eos,)))
        for e in eos_ids:
            if not 0 <= e < vocab:
                raise ConfigError(f"config.json: 'eos_token_id' {e} is outside the vocabulary (0..{vocab - 1})")
        bos = d.get("bos_token_id")
        return cls(vocab=vocab, width=width, layers=tuple(layers), norm_eps=nnum("eps"), postln_alpha=require_float(d, "postln_alpha"),
                   logit_softcap=cap, eos_token_id=eos_ids, bos_token_id=None if bos is None else int(bos),
                   architecture=str(d.get("architecture") or "Burinex"))

    def to_dict(self) -> Dict[str, Any]:
        layers = []
        for layer in self.layers:
            m = layer.mixer
            if layer.type == "attention":
                mixer: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
                if m.q_temp is not None:
                    mixer["q_temp"] = {"coef": m.q_temp.coef, "every": m.q_temp.every}
            elif layer.type == "latent_attention":
                mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
                         "q_rank": m.q_rank, "scale": m.scale}
                if m.window:
                    mixer["mask"] = {"size": m.window}
                if m.rot is not None:
                    mixer["rot"] = {"base": m.rot.base, "dims": m.rot.dims}
                    if m.rot.scaling is not None:
                        s = m.rot.scaling
                        mixer["rot"]["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
            else:
                mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": list(m.decay)}
            mlp = None
            if layer.mlp is not None:
                f = layer.mlp
                mlp = {"kind": "moe", "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.ff}}
                if f.shared_ff:
                    mlp["shared"] = {"ff": f.shared_ff}
            layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                             "norm": {"eps": self.norm_eps}, "postln_alpha": self.postln_alpha, "layers": layers}
        if self.logit_softcap:
            d["logit_softcap"] = self.logit_softcap
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        if self.bos_token_id is not None:
            d["bos_token_id"] = self.bos_token_id
        return d

    @property
    def max_positions(self) -> int:
        return MAX_POSITIONS

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def stop_token_ids(self) -> Tuple[int, ...]:
        return self.eos_token_id

    @property
    def bos_token(self) -> int:
        return self.bos_token_id if self.bos_token_id is not None else 0


register_preset_folder(os.path.join(os.path.dirname(os.path.abspath(__file__)), "presets"))
