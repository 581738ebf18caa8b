"""Typed configuration of the Vekanex decoder, read from its ``config.json``.

The file names the design under ``architecture`` and lists its layers, each with its own mixer and feed-forward::

    {"architecture": "Vekanex", "vocab": V, "width": W, "norm": {"eps": e}, "residual_mult": m, "logit_softcap": c | absent,
     "layers": [
       {"type": "mlstm", "mixer": {"heads": H, "dim": d, "vdim": dv, "gate_cap": c},
        "mlp": {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": k}, "shared": {"ff": F'} | absent} | null},
       {"type": "gla", "mixer": {"heads": H, "dim": d, "vdim": dv, "tau": t}, "mlp": ...},
       {"type": "parallel",
        "mixer": {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": c, "rot": {"dims": n, "base": b}},
                  "right": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "conv": taps},
                  "left_scale": a, "right_scale": b}, "mlp": ...},
       {..., "weights_of": j}]}

``weights_of`` makes an entry one more run of layer j on that layer's tensors, with pages and state of its own; an entry that
says otherwise about its mixer or feed-forward than layer j is refused.  Every size and every constant that differs between
models of the design comes from there; sizes that only a tensor's shape gives (the ranks of the low-rank parts) are read from
the checkpoint's header by the loader, or are given as ``mixer.rank`` (``gla``) and ``mixer.right.decay_rank`` and
``mixer.right.gate_rank`` (``parallel``).
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .llama import ConfigError, _need, _optional
from .zepavik import _positive, _section

ARCHITECTURE = "Vekanex"
MLP_KINDS = ("moe",)


def _rank(raw, key: str, where: str) -> int:
    rank = _optional(raw, key, int, 0)
    if rank < 0:
        raise ConfigError(f"config.json: {where}{key} must not be negative")
    return rank


def _grouped(raw, where: str) -> Tuple[int, int]:
    heads = _positive(_need(raw, "heads", int), where + "heads")
    kv_heads = _positive(_optional(raw, "kv_heads", int, heads), where + "kv_heads")
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    return heads, kv_heads


def _sizes(raw, where: str) -> Tuple[int, int]:
    dim = _positive(_need(raw, "dim", int), where + "dim")
    return dim, _positive(_optional(raw, "vdim", int, dim), where + "vdim")


@dataclass(frozen=True)
class VekanexMlstm:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, raw, where: str) -> "VekanexMlstm":
        heads = _positive(_need(raw, "heads", int), where + "heads")
        cap = _need(raw, "gate_cap", float)
        if not cap > 0.0:
            raise ConfigError(f"config.json: {where}gate_cap must be positive")
        return cls(heads, *_sizes(raw, where), cap)

    def to_dict(self) -> dict:
        return {"dim": self.dim, "gate_cap": self.gate_cap, "heads": self.heads, "vdim": self.vdim}

    def open_ranks(self):
        return {}


@dataclass(frozen=True)
class VekanexGla:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int = 0                    # of the decay's low-rank part; 0: read from the checkpoint (``a1``'s rows)

    @classmethod
    def from_dict(cls, raw, where: str) -> "VekanexGla":
        heads = _positive(_need(raw, "heads", int), where + "heads")
        tau = _need(raw, "tau", float)
        if not tau > 0.0:
            raise ConfigError(f"config.json: {where}tau must be positive")
        return cls(heads, *_sizes(raw, where), tau, _rank(raw, "rank", where))

    def to_dict(self) -> dict:
        raw = {"dim": self.dim, "heads": self.heads, "tau": self.tau, "vdim": self.vdim}
        if self.rank:
            raw["rank"] = self.rank
        return raw

    def open_ranks(self):
        """Field -> the tensor (behind the mixer's prefix) whose rows say it, for the sizes that are still open."""
        return {} if self.rank else {"rank": "a1"}

    def with_ranks(self, ranks) -> "VekanexGla":
        return dataclasses.replace(self, **ranks)


@dataclass(frozen=True)
class VekanexAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int                    # 0: nothing is rotated
    rot_base: float

    @classmethod
    def from_dict(cls, raw, where: str) -> "VekanexAttention":
        heads, kv_heads = _grouped(raw, where)
        dim, vdim = _sizes(raw, where)
        rot = _section(raw, "rot", where, required=False)
        dims, base = 0, 1.0
        if rot is not None:
            dims, base = _need(rot, "dims", int), _need(rot, "base", float)
            if dims < 0 or dims % 2 or dims > dim:
                raise ConfigError(f"config.json: {where}rot.dims ({dims}) must be an even count within a head of {dim} numbers")
            if not base > 0.0:
                raise ConfigError(f"config.json: {where}rot.base must be positive")
        return cls(heads, kv_heads, dim, vdim, _need(raw, "scale", float), dims, base)

    def to_dict(self) -> dict:
        raw = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.rot_dims:
            raw["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        return raw


@dataclass(frozen=True)
class VekanexDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int = 0              # of the low-rank parts; 0: read from the checkpoint (``a1``'s and ``g1``'s rows)
    gate_rank: int = 0

    @classmethod
    def from_dict(cls, raw, where: str) -> "VekanexDelta":
        heads, kv_heads = _grouped(raw, where)
        dim, vdim = _sizes(raw, where)
        return cls(heads, kv_heads, dim, vdim, _positive(_need(raw, "conv", int), where + "conv"),
                   _rank(raw, "decay_rank", where), _rank(raw, "gate_rank", where))

    def to_dict(self) -> dict:
        raw = {"conv": self.taps, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "vdim": self.vdim}
        if self.decay_rank:
            raw["decay_rank"] = self.decay_rank
        if self.gate_rank:
            raw["gate_rank"] = self.gate_rank
        return raw


@dataclass(frozen=True)
class VekanexParallel:
    left: VekanexAttention
    right: VekanexDelta
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, raw, where: str) -> "VekanexParallel":
        return cls(VekanexAttention.from_dict(_section(raw, "left", where), where + "left."),
                   VekanexDelta.from_dict(_section(raw, "right", where), where + "right."),
                   _optional(raw, "left_scale", float, 1.0), _optional(raw, "right_scale", float, 1.0))

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "left_scale": self.left_scale, "right": self.right.to_dict(),
                "right_scale": self.right_scale}

    def open_ranks(self):
        return {field: name for field, name, rank in (("decay_rank", "right.a1", self.right.decay_rank),
                                                      ("gate_rank", "right.g1", self.right.gate_rank)) if not rank}

    def with_ranks(self, ranks) -> "VekanexParallel":
        return dataclasses.replace(self, right=dataclasses.replace(self.right, **ranks))


MIXERS = {"mlstm": VekanexMlstm, "gla": VekanexGla, "parallel": VekanexParallel}


@dataclass(frozen=True)
class VekanexMlp:
    ff: int
    experts: int
    top: int
    shared_ff: int                   # 0: no shared expert

    @classmethod
    def from_dict(cls, raw, where: str) -> "VekanexMlp":
        kind = _optional(raw, "kind", str, "moe")
        if kind not in MLP_KINDS:
            raise ConfigError(f"config.json: {where}kind '{kind}' is not a feed-forward of this design ({', '.join(MLP_KINDS)})")
        expert, router = _section(raw, "expert", where), _section(raw, "router", where)
        experts = _positive(_need(router, "experts", int), where + "router.experts")
        top = _positive(_need(router, "top", int), where + "router.top")
        if top > experts:
            raise ConfigError(f"config.json: {where}router.top ({top}) exceeds router.experts ({experts})")
        shared = _section(raw, "shared", where, required=False)
        shared_ff = _positive(_need(shared, "ff", int), where + "shared.ff") if shared is not None else 0
        return cls(_positive(_need(expert, "ff", int), where + "expert.ff"), experts, top, shared_ff)

    def to_dict(self) -> dict:
        raw = {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            raw["shared"] = {"ff": self.shared_ff}
        return raw


@dataclass(frozen=True)
class VekanexLayer:
    type: str
    mixer: Any                       # VekanexMlstm, VekanexGla or VekanexParallel, by ``type``
    mlp: Optional[VekanexMlp]
    weights_of: Optional[int] = None

    @classmethod
    def from_dict(cls, raw, index: int) -> "VekanexLayer":
        where = f"layers[{index}]."
        if not isinstance(raw, dict):
            raise ConfigError(f"config.json: layers[{index}] must be an object")
        kind = _need(raw, "type", str)
        if kind not in MIXERS:
            raise ConfigError(f"config.json: {where}type '{kind}' is not a mixer of this design ({', '.join(MIXERS)})")
        mixer = MIXERS[kind].from_dict(_section(raw, "mixer", where), where + "mixer.")
        mlp = _section(raw, "mlp", where, required=False)
        owner = None if raw.get("weights_of") is None else _need(raw, "weights_of", int)
        return cls(kind, mixer, VekanexMlp.from_dict(mlp, where + "mlp.") if mlp is not None else None, owner)

    def to_dict(self) -> dict:
        raw = {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp is not None else None}
        if self.weights_of is not None:
            raw["weights_of"] = self.weights_of
        return raw


@dataclass(frozen=True)
class VekanexConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    logit_softcap: float             # 0: logits are not capped
    layers: Tuple[VekanexLayer, ...]
    architecture: str = ARCHITECTURE

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "VekanexConfig":
        vocab = _positive(_need(raw, "vocab", int), "vocab")
        width = _positive(_need(raw, "width", int), "width")
        norm = _section(raw, "norm", "")
        cap = 0.0 if raw.get("logit_softcap") is None else _need(raw, "logit_softcap", float)
        if cap < 0.0:
            raise ConfigError("config.json: logit_softcap must not be negative")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        config = cls(vocab, width, _need(norm, "eps", float), _optional(raw, "residual_mult", float, 1.0), cap,
                     tuple(VekanexLayer.from_dict(layer, i) for i, layer in enumerate(layers)))
        for i, layer in enumerate(config.layers):
            owner = config.layers[config.owner(i)]
            if (layer.type, layer.mixer, layer.mlp) != (owner.type, owner.mixer, owner.mlp):
                raise ConfigError(f"config.json: layers[{i}] uses the weights of layers[{config.owner(i)}] but differs from it")
        return config

    def owner(self, index: int) -> int:
        """The layer whose tensors layer ``index`` uses (itself, unless it says ``weights_of``)."""
        seen = {index}
        while self.layers[index].weights_of is not None:
            index = self.layers[index].weights_of
            if not 0 <= index < len(self.layers) or index in seen:
                raise ConfigError(f"config.json: weights_of {index} names no layer that has weights")
            seen.add(index)
        return index

    def needs_tensor_shapes(self) -> bool:
        """True if a size is still open that only the checkpoint's tensors give."""
        return any(layer.mixer.open_ranks() for layer in self.layers)

    def with_tensor_shapes(self, shapes: Mapping[str, Tuple[int, ...]]) -> "VekanexConfig":
        """The configuration with the sizes that ``config.json`` leaves to the tensors' shapes filled in."""
        layers = []
        for i, layer in enumerate(self.layers):
            ranks = {}
            for field, tensor in layer.mixer.open_ranks().items():
                name = f"l{self.owner(i)}.mix.{tensor}"
                shape = shapes.get(name)
                if shape is None or len(shape) != 2 or shape[0] <= 0:
                    raise ConfigError(f"the checkpoint has no matrix '{name}' to read a low-rank part's rank from")
                ranks[field] = int(shape[0])
            layers.append(dataclasses.replace(layer, mixer=layer.mixer.with_ranks(ranks)) if ranks else layer)
        return dataclasses.replace(self, layers=tuple(layers))

    def to_dict(self) -> dict:
        raw = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "residual_mult": self.residual_mult, "layers": [layer.to_dict() for layer in self.layers]}
        if self.logit_softcap:
            raw["logit_softcap"] = self.logit_softcap
        return raw
