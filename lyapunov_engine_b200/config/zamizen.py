"""ZamizenConfig: the keys of a Zamizen checkpoint's config.json, typed.

    {"architecture": "Zamizen", "vocab": V, "width": W, "norm": {"eps": ..}, "residual_mult": m,
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "conv", "kv_from",
                           "rot": {"dims", "base"}}, "mlp": ..}
                | {"type": "latent_attention",
                   "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale",
                             "rot": {"dims", "base", "scaling": {"factor", "original", "fast", "slow"}}}, "mlp": ..}, ...]}
    mlp: {"kind": "dense", "ff"} | null

Every size and constant a layer uses is read from its own entry; nothing has a
default.  Keys that may be absent, and what their absence means: an attention
layer's ``kv_from`` (keys and values of its own), a rotation's ``scaling`` (the
plain rates), ``mlp`` null (a layer without feed-forward).
"""
from __future__ import annotations

from dataclasses import dataclass

from .base import ConfigError, KeyReader


@dataclass(frozen=True)
class RampedScaling:
    factor: float
    original: float
    fast: float
    slow: float

    def as_dict(self) -> dict:
        return {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class ZamizenAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    taps: int
    rot_dims: int
    rot_base: float
    kv_from: int | None      # the layer whose keys and values it reads (None: its own)


@dataclass(frozen=True)
class ZamizenLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    scaling: RampedScaling | None


@dataclass(frozen=True)
class ZamizenLayer:
    mixer: ZamizenAttention | ZamizenLatent
    ff: int                  # 0: no feed-forward


def _attention(m: KeyReader) -> ZamizenAttention:
    rot = KeyReader(m.mapping("rot"), m.source + ".rot")
    a = ZamizenAttention(heads=m.integer("heads"), kv_heads=m.integer("kv_heads"), dim=m.integer("dim"), vdim=m.integer("vdim"),
                         scale=m.number("scale", positive=False), taps=m.integer("conv"),
                         rot_dims=rot.integer("dims", minimum=0), rot_base=rot.number("base"),
                         kv_from=m.integer("kv_from", None, minimum=0))
    if a.heads % a.kv_heads:
        raise ConfigError(f"{m.source}: {a.heads} heads do not divide into {a.kv_heads} kv_heads")
    if a.rot_dims % 2 or a.rot_dims > a.dim:
        raise ConfigError(f"{rot.source}: dims {a.rot_dims} must be even and at most dim {a.dim}")
    if rot.raw.get("scaling") is not None:
        raise ConfigError(f"{rot.source}: an attention layer's rotation has no 'scaling'")
    return a


def _latent(m: KeyReader) -> ZamizenLatent:
    rot = KeyReader(m.mapping("rot"), m.source + ".rot")
    scaling = rot.mapping("scaling", None)
    if scaling is not None:
        r = KeyReader(scaling, rot.source + ".scaling")
        scaling = RampedScaling(r.number("factor"), r.number("original"), r.number("fast"), r.number("slow"))
    a = ZamizenLatent(heads=m.integer("heads"), dim=m.integer("dim"), rot_dim=m.integer("rot_dim", minimum=0),
                      vdim=m.integer("vdim"), kv_rank=m.integer("kv_rank"), scale=m.number("scale", positive=False),
                      rot_base=rot.number("base"), scaling=scaling)
    if rot.integer("dims", minimum=0) != a.rot_dim or a.rot_dim % 2:
        raise ConfigError(f"{m.source}: rot.dims must equal rot_dim {a.rot_dim} and be even")
    return a


@dataclass(frozen=True)
class ZamizenConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: tuple[ZamizenLayer, ...]
    raw: dict

    @staticmethod
    def from_dict(raw: dict, source: str = "config.json") -> "ZamizenConfig":
        r = KeyReader(raw, source)
        norm = KeyReader(r.mapping("norm"), source + ": norm")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError(f"{source}: 'layers' must be a non-empty list")
        readers = {"attention": _attention, "latent_attention": _latent}
        layers = []
        for i, entry in enumerate(entries):
            where = f"{source}: layers[{i}]"
            if not isinstance(entry, dict):
                raise ConfigError(f"{where} must be an object")
            e = KeyReader(entry, where)
            kind = e.string("type")
            if kind not in readers:
                raise ConfigError(f"{where}: unknown layer type {kind!r} (known: {', '.join(map(repr, sorted(readers)))})")
            mixer = readers[kind](KeyReader(e.mapping("mixer"), where + ".mixer"))
            if kind == "attention" and mixer.kv_from is not None:
                source_layer = layers[mixer.kv_from].mixer if mixer.kv_from < i else None
                if not isinstance(source_layer, ZamizenAttention) or source_layer.kv_from is not None:
                    raise ConfigError(f"{where}.mixer: kv_from {mixer.kv_from} is not an earlier attention layer with keys of its own")
                if ((source_layer.kv_heads, source_layer.dim, source_layer.vdim) != (mixer.kv_heads, mixer.dim, mixer.vdim)):
                    raise ConfigError(f"{where}.mixer: layer {mixer.kv_from}, whose keys it reads, has other kv_heads, dim or vdim")
            ff = 0
            if entry.get("mlp") is not None:
                f = KeyReader(e.mapping("mlp"), where + ".mlp")
                ff_kind = f.string("kind")
                if ff_kind != "dense":
                    raise ConfigError(f"{where}.mlp: unknown kind {ff_kind!r} (known: 'dense')")
                ff = f.integer("ff")
            layers.append(ZamizenLayer(mixer, ff))
        return ZamizenConfig(architecture=r.string("architecture"), vocab=r.integer("vocab"), width=r.integer("width"),
                             norm_eps=norm.number("eps"), residual_mult=r.number("residual_mult", positive=False),
                             layers=tuple(layers), raw=dict(raw))
