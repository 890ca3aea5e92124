"""Typed configuration of the Gevipel decoder, read from its config.json keys.

A Gevipel model is a list of layers; each layer names its mixer (`type`: "delta", "attention" or "latent_attention"),
gives the mixer's sizes and constants (`mixer`) and its feed-forward (`mlp`, or null for a layer without one).  A stretch
of the layers may run several times in a row with the same weights (`loop`).

    architecture      "Gevipel"
    vocab, width      vocabulary and residual width (the head has its own matrix)
    embedding.scale   what the embedding's rows are multiplied by
    norm.eps          epsilon of every norm (layer norms with weight and bias; the RMS norms inside the mixers)
    residual_mult     multiplier on every branch as it joins the stream
    layers[i]         {"type", "mixer": {...}, "mlp": {...} | null}
    loop              {"start", "stop", "times"}: layers start .. stop - 1 run `times` times; absent: every layer once

delta:             `heads`, `kv_heads`, `dim`, `vdim`, `conv` (taps of the convolution).
attention:         `heads`, `kv_heads`, `dim`, `vdim` (the keys' size: the values are the keys), `scale`, `mask.size` (a sliding
                   window; absent: every earlier position), `q_temp` = {"coef", "every"} (absent: none).
latent_attention:  `heads`, `dim` (unrotated query/key size of a head), `rot_dim` (rotated size), `vdim`, `kv_rank`, `scale`,
                   `rot` = {"dims", "base"} (interleaved pairs over the whole rotated part).
mlp:               {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}}.
"""
from __future__ import annotations

from dataclasses import dataclass

from .base import ConfigError, KeyReader, read_config_json
from .lavutar import Loop
from .zoporax import _object

MIXERS = ("delta", "attention", "latent_attention")


@dataclass(frozen=True)
class Experts:
    ff: int                            # an expert's hidden size
    experts: int
    top: int

    @classmethod
    def from_dict(cls, data, where: str) -> "Experts | None":
        if data is None:
            return None
        if not isinstance(data, dict):
            raise ConfigError(f"{where}: 'mlp' must be an object or null")
        where = f"{where}.mlp"
        kind = KeyReader(data, where).string("kind", "moe")
        if kind != "moe":
            raise ConfigError(f"{where}: kind {kind!r} is not supported (supported: 'moe')")
        ff = KeyReader(_object(data, "expert", where), f"{where}.expert").integer("ff", minimum=1)
        r = KeyReader(_object(data, "router", where), f"{where}.router")
        experts, top = r.integer("experts", minimum=1), r.integer("top", minimum=1)
        if top > experts:
            raise ConfigError(f"{where}.router: 'top' {top} exceeds the {experts} experts")
        return cls(ff=ff, experts=experts, top=top)

    def to_dict(self) -> dict:
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


def _heads(mixer: dict, where: str) -> dict:
    m = KeyReader(mixer, where)
    heads = m.integer("heads", minimum=1)
    kv_heads = m.integer("kv_heads", heads, minimum=1)
    if heads % kv_heads:
        raise ConfigError(f"{where}: {heads} heads are not a multiple of {kv_heads} kv_heads")
    dim = m.integer("dim", minimum=1)
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": m.integer("vdim", dim, minimum=1)}


@dataclass(frozen=True)
class DeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @classmethod
    def from_dict(cls, mixer: dict, where: str) -> "DeltaMixer":
        return cls(**_heads(mixer, where), conv=KeyReader(mixer, where).integer("conv", minimum=1))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int | None = None
    temp_coef: float | None = None       # q times 1 + coef ln(floor((p + 1) / every) + 1)
    temp_every: int | None = None

    @classmethod
    def from_dict(cls, mixer: dict, where: str) -> "AttentionMixer":
        sizes = _heads(mixer, where)
        if sizes["vdim"] != sizes["dim"]:
            raise ConfigError(f"{where}: 'vdim' {sizes['vdim']} is not 'dim' {sizes['dim']} (the values are the keys)")
        more = {}
        mask = _object(mixer, "mask", where, required=False)
        if mask is not None:
            more["window"] = KeyReader(mask, f"{where}.mask").integer("size", None, minimum=1)
        qt = _object(mixer, "q_temp", where, required=False)
        if qt is not None:
            t = KeyReader(qt, f"{where}.q_temp")
            more.update(temp_coef=t.number("coef"), temp_every=t.integer("every", minimum=1))
        return cls(**sizes, scale=KeyReader(mixer, where).number("scale", sizes["dim"] ** -0.5), **more)

    @property
    def slopes(self) -> tuple[float, ...]:
        """What head h's score loses per position of distance: 2^(-8 (h + 1) / heads)."""
        return tuple(2.0 ** (-8.0 * (h + 1) / self.heads) for h in range(self.heads))

    def to_dict(self) -> dict:
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.window is not None:
            out["mask"] = {"size": self.window}
        if self.temp_coef is not None:
            out["q_temp"] = {"coef": self.temp_coef, "every": self.temp_every}
        return out


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_dims: int | None = None          # rotated dimensions and base; None: the rotated part is used as it comes
    rot_base: float | None = None

    @classmethod
    def from_dict(cls, mixer: dict, where: str) -> "LatentMixer":
        m = KeyReader(mixer, where)
        dim, rot_dim = m.integer("dim", minimum=1), m.integer("rot_dim", minimum=0)
        more = {}
        rot = _object(mixer, "rot", where, required=False)
        if rot is not None and rot_dim:
            r = KeyReader(rot, f"{where}.rot")
            dims = r.integer("dims", rot_dim, minimum=0)
            if dims % 2 or dims > rot_dim:
                raise ConfigError(f"{where}.rot: 'dims' {dims} must be even and at most the rotated size {rot_dim}")
            if dims:
                more.update(rot_dims=dims, rot_base=r.number("base", positive=True))
        return cls(heads=m.integer("heads", minimum=1), dim=dim, rot_dim=rot_dim, vdim=m.integer("vdim", dim, minimum=1),
                   kv_rank=m.integer("kv_rank", minimum=1), scale=m.number("scale", (dim + rot_dim) ** -0.5), **more)

    def to_dict(self) -> dict:
        out = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank, "scale": self.scale}
        if self.rot_dims is not None:
            out["rot"] = {"dims": self.rot_dims, "base": self.rot_base}
        return out


_MIXER_OF = {"delta": DeltaMixer, "attention": AttentionMixer, "latent_attention": LatentMixer}


@dataclass(frozen=True)
class GevipelLayer:
    type: str
    mixer: DeltaMixer | AttentionMixer | LatentMixer
    mlp: Experts | None

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


def _layer(i: int, data) -> GevipelLayer:
    where = f"config.json: layers[{i}]"
    if not isinstance(data, dict):
        raise ConfigError(f"{where} must be an object")
    kind = KeyReader(data, where).string("type")
    if kind not in MIXERS:
        raise ConfigError(f"{where}: type {kind!r} is not one of {', '.join(MIXERS)}")
    return GevipelLayer(type=kind, mixer=_MIXER_OF[kind].from_dict(_object(data, "mixer", where), f"{where}.mixer"),
                        mlp=Experts.from_dict(data.get("mlp"), where))


@dataclass(frozen=True)
class GevipelConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[GevipelLayer, ...]
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    loop: Loop | None = None
    max_positions: int = 32768           # no key of the design bounds a sequence; this sizes tables and default caches
    architectures: tuple[str, ...] = ("Gevipel",)

    @classmethod
    def from_dict(cls, data: dict) -> "GevipelConfig":
        r = KeyReader(data)
        layers = data.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        loop = None
        ld = _object(data, "loop", "config.json", required=False)
        if ld is not None:
            loop = Loop.from_dict(ld, len(layers))
        emb = _object(data, "embedding", "config.json", required=False)
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                   norm_eps=KeyReader(_object(data, "norm", "config.json"), "config.json: norm").number("eps", positive=True),
                   layers=tuple(_layer(i, layer) for i, layer in enumerate(layers)),
                   embedding_scale=KeyReader(emb, "config.json: embedding").number("scale", 1.0) if emb is not None else 1.0,
                   residual_mult=r.number("residual_mult", 1.0), loop=loop, max_positions=r.integer("max_positions", 32768, minimum=1))

    @classmethod
    def from_json(cls, folder_or_file) -> "GevipelConfig":
        return cls.from_dict(read_config_json(folder_or_file))

    def runs(self) -> list[tuple[int, bool]]:
        """(layer, whether a pass of the loop other than the first starts with it) for every run of a layer, in order."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        lo, hi = self.loop.start, self.loop.stop
        runs = [(i, False) for i in range(lo)]
        for turn in range(self.loop.times):
            runs += [(i, turn > 0 and i == lo) for i in range(lo, hi)]
        return runs + [(i, False) for i in range(hi, n)]

    def to_dict(self) -> dict:
        out = {"architecture": "Gevipel", "vocab": self.vocab, "width": self.width, "embedding": {"scale": self.embedding_scale},
               "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "layers": [layer.to_dict() for layer in self.layers]}
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        if self.max_positions != 32768:
            out["max_positions"] = self.max_positions
        return out
