"""Typed configuration of the Tobozen decoder, read from its ``config.json``.

The file names the design under ``architecture`` and lists its layers, each with its own mixer and feed-forward::

    {"architecture": "Tobozen", "vocab": V, "width": W, "norm": {"eps": e, "groups": g},
     "layers": [
       {"type": "attention",
        "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": c, "rot": {"dims": n, "base": b},
                  "v_mix": true | false},
        "mlp": {"kind": "moe", "expert": {"ff": F, "limit": c}, "router": {"experts": E, "top": k}} | null},
       {"type": "mamba2",
        "mixer": {"heads": H, "vdim": dv, "state": N, "groups": G, "conv": taps, "norm_groups": m}, "mlp": ...},
       {"type": "lightning",
        "mixer": {"heads": H, "dim": d, "vdim": dv, "decay": [one number per head]}, "mlp": ...}]}

Every size and every constant that differs between models of the design comes from there; layers may differ from one
another in all of their numbers.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .llama import ConfigError, _need, _optional
from .zepavik import _positive, _section

ARCHITECTURE = "Tobozen"
MLP_KINDS = ("moe",)


@dataclass(frozen=True)
class TobozenAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int                    # 0: nothing is rotated
    rot_base: float
    v_mix: bool

    @classmethod
    def from_dict(cls, raw, where: str) -> "TobozenAttention":
        heads = _positive(_need(raw, "heads", int), where + "heads")
        kv_heads = _positive(_optional(raw, "kv_heads", int, heads), where + "kv_heads")
        if heads % kv_heads:
            raise ConfigError(f"config.json: {where}heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
        dim = _positive(_need(raw, "dim", int), where + "dim")
        vdim = _positive(_optional(raw, "vdim", int, dim), where + "vdim")
        rot = _section(raw, "rot", where, required=False)
        dims, base = 0, 1.0
        if rot is not None:
            dims, base = _need(rot, "dims", int), _need(rot, "base", float)
            if dims < 0 or dims % 2 or dims > dim:
                raise ConfigError(f"config.json: {where}rot.dims ({dims}) must be an even count within a head of {dim} numbers")
            if not base > 0.0:
                raise ConfigError(f"config.json: {where}rot.base must be positive")
        scale = _need(raw, "scale", float)
        if not scale > 0.0:
            raise ConfigError(f"config.json: {where}scale must be positive")
        v_mix = raw.get("v_mix", False)
        if not isinstance(v_mix, bool):
            raise ConfigError(f"config.json: {where}v_mix must be true or false")
        return cls(heads, kv_heads, dim, vdim, scale, dims, base, v_mix)

    def to_dict(self) -> dict:
        raw = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "v_mix": self.v_mix,
               "vdim": self.vdim}
        if self.rot_dims:
            raw["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        return raw


@dataclass(frozen=True)
class TobozenMamba2:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int

    @classmethod
    def from_dict(cls, raw, where: str) -> "TobozenMamba2":
        heads = _positive(_need(raw, "heads", int), where + "heads")
        vdim = _positive(_need(raw, "vdim", int), where + "vdim")
        groups = _positive(_optional(raw, "groups", int, 1), where + "groups")
        if heads % groups:
            raise ConfigError(f"config.json: {where}heads ({heads}) must be a multiple of groups ({groups})")
        norm_groups = _positive(_optional(raw, "norm_groups", int, 1), where + "norm_groups")
        if heads * vdim % norm_groups:
            raise ConfigError(f"config.json: {where}norm_groups ({norm_groups}) must divide heads * vdim ({heads * vdim})")
        return cls(heads, vdim, _positive(_need(raw, "state", int), where + "state"), groups,
                   _positive(_need(raw, "conv", int), where + "conv"), norm_groups)

    def to_dict(self) -> dict:
        return {"conv": self.taps, "groups": self.groups, "heads": self.heads, "norm_groups": self.norm_groups,
                "state": self.state, "vdim": self.vdim}


@dataclass(frozen=True)
class TobozenLightning:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    @classmethod
    def from_dict(cls, raw, where: str) -> "TobozenLightning":
        heads = _positive(_need(raw, "heads", int), where + "heads")
        dim = _positive(_need(raw, "dim", int), where + "dim")
        decay = raw.get("decay")
        if (not isinstance(decay, list) or len(decay) != heads
                or not all(isinstance(d, (int, float)) and not isinstance(d, bool) and 0.0 <= d <= 1.0 for d in decay)):
            raise ConfigError(f"config.json: {where}decay must list one number between 0 and 1 for each of the {heads} heads")
        return cls(heads, dim, _positive(_optional(raw, "vdim", int, dim), where + "vdim"), tuple(float(d) for d in decay))

    def to_dict(self) -> dict:
        return {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}


MIXERS = {"attention": TobozenAttention, "mamba2": TobozenMamba2, "lightning": TobozenLightning}


@dataclass(frozen=True)
class TobozenMlp:
    ff: int
    limit: float                     # both branches of an expert are clamped to it
    experts: int
    top: int

    @classmethod
    def from_dict(cls, raw, where: str) -> "TobozenMlp":
        kind = _optional(raw, "kind", str, "moe")
        if kind not in MLP_KINDS:
            raise ConfigError(f"config.json: {where}kind '{kind}' is not a feed-forward of this design ({', '.join(MLP_KINDS)})")
        expert, router = _section(raw, "expert", where), _section(raw, "router", where)
        limit = _need(expert, "limit", float)
        if not limit > 0.0:
            raise ConfigError(f"config.json: {where}expert.limit must be positive")
        experts = _positive(_need(router, "experts", int), where + "router.experts")
        top = _positive(_need(router, "top", int), where + "router.top")
        if top > experts:
            raise ConfigError(f"config.json: {where}router.top ({top}) exceeds router.experts ({experts})")
        return cls(_positive(_need(expert, "ff", int), where + "expert.ff"), limit, experts, top)

    def to_dict(self) -> dict:
        return {"expert": {"ff": self.ff, "limit": self.limit}, "kind": "moe",
                "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class TobozenLayer:
    type: str
    mixer: Any                       # TobozenAttention, TobozenMamba2 or TobozenLightning, by ``type``
    mlp: Optional[TobozenMlp]

    @classmethod
    def from_dict(cls, raw, index: int) -> "TobozenLayer":
        where = f"layers[{index}]."
        if not isinstance(raw, dict):
            raise ConfigError(f"config.json: layers[{index}] must be an object")
        kind = _need(raw, "type", str)
        if kind not in MIXERS:
            raise ConfigError(f"config.json: {where}type '{kind}' is not a mixer of this design ({', '.join(MIXERS)})")
        mixer = MIXERS[kind].from_dict(_section(raw, "mixer", where), where + "mixer.")
        mlp = _section(raw, "mlp", where, required=False)
        return cls(kind, mixer, TobozenMlp.from_dict(mlp, where + "mlp.") if mlp is not None else None)

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp is not None else None}


@dataclass(frozen=True)
class TobozenConfig:
    vocab: int
    width: int
    norm_eps: float
    norm_groups: int
    layers: Tuple[TobozenLayer, ...]
    architecture: str = ARCHITECTURE

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "TobozenConfig":
        vocab = _positive(_need(raw, "vocab", int), "vocab")
        width = _positive(_need(raw, "width", int), "width")
        norm = _section(raw, "norm", "")
        groups = _positive(_optional(norm, "groups", int, 1), "norm.groups")
        if width % groups:
            raise ConfigError(f"config.json: norm.groups ({groups}) must divide width ({width})")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        parsed = tuple(TobozenLayer.from_dict(layer, i) for i, layer in enumerate(layers))
        mixing = [layer.mixer for layer in parsed if layer.type == "attention" and layer.mixer.v_mix]
        if any(m.kv_heads * m.vdim != mixing[0].kv_heads * mixing[0].vdim for m in mixing):
            raise ConfigError("config.json: layers that mix values (v_mix) must have equally many value numbers (kv_heads * vdim)")
        return cls(vocab, width, _need(norm, "eps", float), groups, parsed)

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps, "groups": self.norm_groups},
                "layers": [layer.to_dict() for layer in self.layers]}
