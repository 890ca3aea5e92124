"""Typed configuration of the Korazen decoder, read from its config.json keys.

A Korazen model is a list of layers; each layer names its mixer (`type`: "channel_delta" or "parallel"), gives the
mixer's sizes and constants (`mixer`) and its feed-forward (`mlp`, or null for a layer without one).

    architecture   "Korazen"
    vocab, width   vocabulary and residual width (the head has its own matrix)
    norm.eps       epsilon of every norm
    logit_scale    what the logits are multiplied by
    layers[i]      {"type", "mixer": {...}, "mlp": {...} | null}

channel_delta: `heads`, `kv_heads` (heads of q and k; absent: as many as `heads`), `dim`, `vdim`, `conv` (taps of the
               convolutions); optional `rank` and `gate_rank`, the inner sizes of the decays' and the output gate's two
               products (absent: the sizes the stored tensors have; random weights need the keys).
parallel:      `left` = {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"} | absent (every earlier position),
               "rot": {"dims", "base"} | absent}, `right` = {"heads", "dim", "vdim", "decay": one number per head}.
mlp:           {"kind": "dense", "ff", "limit"}.
"""
from __future__ import annotations

from dataclasses import dataclass

from .base import ConfigError, KeyReader, read_config_json
from .zoporax import _object

MIXERS = ("channel_delta", "parallel")


@dataclass(frozen=True)
class KorazenFeedForward:
    ff: int
    limit: float

    @classmethod
    def from_dict(cls, data, where: str) -> "KorazenFeedForward | None":
        if data is None:
            return None
        if not isinstance(data, dict):
            raise ConfigError(f"{where}: 'mlp' must be an object or null")
        r = KeyReader(data, f"{where}.mlp")
        kind = r.string("kind", "dense")
        if kind != "dense":
            raise ConfigError(f"{where}.mlp: kind {kind!r} is not supported (supported: 'dense')")
        return cls(ff=r.integer("ff", minimum=1), limit=r.number("limit", positive=True))

    def to_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class DeltaHeads:
    """Gated delta rule: a matrix state per value head, key channels that decay each at their own rate."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    rank: int | None = None
    gate_rank: int | None = None

    @classmethod
    def from_dict(cls, mixer: dict, where: str) -> "DeltaHeads":
        m = KeyReader(mixer, where)
        heads = m.integer("heads", minimum=1)
        kv_heads = m.integer("kv_heads", heads, minimum=1)
        if heads % kv_heads:
            raise ConfigError(f"{where}: {heads} heads are not a multiple of {kv_heads} kv_heads")
        dim = m.integer("dim", minimum=1)
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, vdim=m.integer("vdim", dim, minimum=1), conv=m.integer("conv", minimum=1),
                   rank=m.integer("rank", None, minimum=1), gate_rank=m.integer("gate_rank", None, minimum=1))

    def to_dict(self) -> dict:
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}
        if self.rank is not None:
            out["rank"] = self.rank
        if self.gate_rank is not None:
            out["gate_rank"] = self.gate_rank
        return out


@dataclass(frozen=True)
class BlockHeads:
    """Left side of "parallel": grouped softmax attention inside blocks of positions."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    block: int | None = None           # mask.size
    rot_dims: int = 0
    rot_base: float | None = None

    @classmethod
    def from_dict(cls, mixer: dict, where: str) -> "BlockHeads":
        m = KeyReader(mixer, where)
        heads = m.integer("heads", minimum=1)
        kv_heads = m.integer("kv_heads", heads, minimum=1)
        if heads % kv_heads:
            raise ConfigError(f"{where}: {heads} heads are not a multiple of {kv_heads} kv_heads")
        dim = m.integer("dim", minimum=1)
        mask = _object(mixer, "mask", where, required=False)
        rot = _object(mixer, "rot", where, required=False)
        dims, base = 0, None
        if rot is not None:
            r = KeyReader(rot, f"{where}.rot")
            dims = r.integer("dims", dim, minimum=0)
            if dims % 2 or dims > dim:
                raise ConfigError(f"{where}.rot: 'dims' {dims} must be even and at most 'dim' {dim}")
            base = r.number("base", positive=True)
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, vdim=m.integer("vdim", dim, minimum=1), scale=m.number("scale", dim ** -0.5),
                   block=KeyReader(mask, f"{where}.mask").integer("size", None, minimum=1) if mask is not None else None,
                   rot_dims=dims, rot_base=base if dims else None)

    def to_dict(self) -> dict:
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.block is not None:
            out["mask"] = {"size": self.block}
        if self.rot_dims:
            out["rot"] = {"dims": self.rot_dims, "base": self.rot_base}
        return out


@dataclass(frozen=True)
class FixedDecayHeads:
    """Right side of "parallel": a matrix state per head that decays by the head's own constant."""
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]

    @classmethod
    def from_dict(cls, mixer: dict, where: str) -> "FixedDecayHeads":
        m = KeyReader(mixer, where)
        heads, dim = m.integer("heads", minimum=1), m.integer("dim", minimum=1)
        decay = mixer.get("decay")
        if not isinstance(decay, list) or len(decay) != heads or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
            raise ConfigError(f"{where}: 'decay' must be a list of {heads} numbers, one per head, found {decay!r}")
        return cls(heads=heads, dim=dim, vdim=m.integer("vdim", dim, minimum=1), decay=tuple(float(d) for d in decay))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


@dataclass(frozen=True)
class KorazenLayer:
    type: str
    mlp: KorazenFeedForward | None
    delta: DeltaHeads | None = None          # "channel_delta"
    left: BlockHeads | None = None           # "parallel"
    right: FixedDecayHeads | None = None

    def to_dict(self) -> dict:
        m = self.delta.to_dict() if self.type == "channel_delta" else {"left": self.left.to_dict(), "right": self.right.to_dict()}
        return {"type": self.type, "mixer": m, "mlp": None if self.mlp is None else self.mlp.to_dict()}


def _layer(i: int, data) -> KorazenLayer:
    where = f"config.json: layers[{i}]"
    if not isinstance(data, dict):
        raise ConfigError(f"{where} must be an object")
    kind = KeyReader(data, where).string("type")
    if kind not in MIXERS:
        raise ConfigError(f"{where}: type {kind!r} is not one of {', '.join(MIXERS)}")
    mixer = _object(data, "mixer", where)
    mlp = KorazenFeedForward.from_dict(data.get("mlp"), where)
    where = f"{where}.mixer"
    if kind == "channel_delta":
        return KorazenLayer(type=kind, mlp=mlp, delta=DeltaHeads.from_dict(mixer, where))
    return KorazenLayer(type=kind, mlp=mlp, left=BlockHeads.from_dict(_object(mixer, "left", where), f"{where}.left"),
                        right=FixedDecayHeads.from_dict(_object(mixer, "right", where), f"{where}.right"))


@dataclass(frozen=True)
class KorazenConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[KorazenLayer, ...]
    logit_scale: float = 1.0
    max_positions: int = 32768           # no key of the design bounds a sequence; this sizes tables and default caches
    architectures: tuple[str, ...] = ("Korazen",)

    @classmethod
    def from_dict(cls, data: dict) -> "KorazenConfig":
        r = KeyReader(data)
        norm = _object(data, "norm", "config.json")
        layers = data.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                   norm_eps=KeyReader(norm, "config.json: norm").number("eps", positive=True),
                   layers=tuple(_layer(i, layer) for i, layer in enumerate(layers)), logit_scale=r.number("logit_scale", 1.0),
                   max_positions=r.integer("max_positions", 32768, minimum=1))

    @classmethod
    def from_json(cls, folder_or_file) -> "KorazenConfig":
        return cls.from_dict(read_config_json(folder_or_file))

    def to_dict(self) -> dict:
        out = {"architecture": "Korazen", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "logit_scale": self.logit_scale, "layers": [layer.to_dict() for layer in self.layers]}
        if self.max_positions != 32768:
            out["max_positions"] = self.max_positions
        return out
