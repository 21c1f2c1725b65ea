"""Typed configuration of the Bobasun decoder, read from its own ``config.json`` keys.

    {"architecture": "Bobasun", "vocab": V, "width": W, "streams": s, "norm": {"eps": e}, "embedding": {"scale": c},
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "v_mix",
                           "rot": {"base", "dims", "scaling": {"factor"}}},
                 "mlp": {"kind": "dense", "ff", "limit"}}, ...]}

Every size and constant is read from there, layer by layer; nothing is the same for two layers unless the file says so.
``streams``: how many residual streams run side by side.  ``v_mix``: this layer's values are mixed with those of the first
layer that has it.  ``mlp`` may be null (no feed-forward).
"""
from __future__ import annotations

import os
from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, ModelConfig, require_int
from .registry import register_preset_folder
from .vabelorn import _obj, _sub
from .zonevik import _heads

# The file gives no longest sequence; position tables are made for what the engine is asked to hold, up to this.
MAX_POSITIONS = 1 << 17


@dataclass(frozen=True)
class MixedValueAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    v_mix: bool
    rot_base: float
    rot_dims: int           # 0: no rotation
    rot_factor: float       # every frequency is divided by it


@dataclass(frozen=True)
class ClampedFf:
    ff: int
    limit: float


@dataclass(frozen=True)
class BobasunLayer:
    type: str                       # "attention"
    mixer: MixedValueAttention
    mlp: Optional[ClampedFf]


def _mlp(d: Any, where: str) -> Optional[ClampedFf]:
    if d is None:
        return None
    d = _obj(d, where)
    kind = d.get("kind", "dense")
    if kind != "dense":
        raise ConfigError(f"config.json: {where}: 'kind' must be 'dense', got {kind!r}")
    whole, num = _sub(d, where)
    return ClampedFf(ff=whole("ff"), limit=num("limit"))


@dataclass(frozen=True)
class BobasunConfig(ModelConfig):
    vocab: int
    width: int
    layers: Tuple[BobasunLayer, ...]
    norm_eps: float
    streams: int = 1
    embedding_scale: float = 1.0
    eos_token_id: Tuple[int, ...] = ()
    bos_token_id: Optional[int] = None
    architecture: str = field(default="Bobasun")

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "BobasunConfig":
        vocab = require_int(d, "vocab")
        width = require_int(d, "width")
        streams = require_int(d, "streams", default=1)
        _, nnum = _sub(_obj(d.get("norm"), "'norm'"), "'norm'")
        eps = nnum("eps")
        scale = 1.0
        if isinstance(d.get("embedding"), dict) and d["embedding"].get("scale") is not None:
            _, enum = _sub(d["embedding"], "'embedding'")
            scale = enum("scale")
        raw = d.get("layers")
        if not isinstance(raw, (list, tuple)) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        mixed = None        # (layer, kv_heads, vdim) of the first layer whose values the others take in
        for i, entry in enumerate(raw):
            where = f"layers[{i}]"
            entry = _obj(entry, where)
            kind = entry.get("type", "attention")
            if kind != "attention":
                raise ConfigError(f"config.json: {where}: 'type' must be 'attention', got {kind!r}")
            mw = where + ".mixer"
            m = _obj(entry.get("mixer"), mw)
            whole, num, heads, kv, dim = _heads(m, mw)
            vdim = whole("vdim", default=dim)
            base, dims, factor = 10000.0, 0, 1.0
            rot = m.get("rot")
            if rot:
                rwhole, rnum = _sub(_obj(rot, mw + ".rot"), mw + ".rot")
                dims = rwhole("dims", minimum=0)
                if dims % 2 or dims > dim:
                    raise ConfigError(f"config.json: {mw}.rot: 'dims' must be even and at most the head size {dim}, got {dims}")
                base = rnum("base")
                if rot.get("scaling"):
                    _, snum = _sub(_obj(rot["scaling"], mw + ".rot.scaling"), mw + ".rot.scaling")
                    factor = snum("factor")
            v_mix = m.get("v_mix", False)
            if not isinstance(v_mix, bool):
                raise ConfigError(f"config.json: {mw}: 'v_mix' must be true or false, got {v_mix!r}")
            if v_mix:
                if mixed is None:
                    mixed = (i, kv, vdim)
                elif mixed[1:] != (kv, vdim):
                    raise ConfigError(f"config.json: {mw}: 'v_mix' mixes {kv} x {vdim} values with the {mixed[1]} x {mixed[2]} values of "
                                      f"layers[{mixed[0]}]")
            layers.append(BobasunLayer(type=kind, mixer=MixedValueAttention(
                heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=num("scale"), v_mix=v_mix, rot_base=base, rot_dims=dims,
                rot_factor=factor), mlp=_mlp(entry.get("mlp"), where + ".mlp")))
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else (eos,)))
        for e in eos_ids:
            if not 0 <= e < vocab:
                raise ConfigError(f"config.json: 'eos_token_id' {e} is outside the vocabulary (0..{vocab - 1})")
        bos = d.get("bos_token_id")
        return cls(vocab=vocab, width=width, layers=tuple(layers), norm_eps=eps, streams=streams, embedding_scale=scale,
                   eos_token_id=eos_ids, bos_token_id=None if bos is None else int(bos),
                   architecture=str(d.get("architecture") or "Bobasun"))

    def to_dict(self) -> Dict[str, Any]:
        layers = []
        for layer in self.layers:
            m = layer.mixer
            mixer: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                                     "v_mix": m.v_mix}
            if m.rot_dims:
                mixer["rot"] = {"base": m.rot_base, "dims": m.rot_dims}
                if m.rot_factor != 1.0:
                    mixer["rot"]["scaling"] = {"factor": m.rot_factor}
            mlp = None if layer.mlp is None else {"kind": "dense", "ff": layer.mlp.ff, "limit": layer.mlp.limit}
            layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
                             "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale}, "layers": layers}
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
