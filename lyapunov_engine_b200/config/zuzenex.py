"""ZuzenexConfig: the keys of a Zuzenex checkpoint's config.json, typed.

    {"architecture": "Zuzenex", "vocab": V, "width": W, "norm": {"eps": ..},
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "lightning", "mixer": {"heads", "dim", "vdim", "decay": [one per head]}, "mlp": ..}
                | {"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale",
                                                  "q_temp": {"coef", "every"}}, "mlp": ..}, ...]}
    mlp: {"kind": "dense", "ff"}
       | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "identity", "top"}, "shared": {"ff"}}
       | null

Every size and constant a layer uses is read from its own entry; nothing has a
default.  Keys that may be absent, and what their absence means: ``loop``
(every layer runs once), a mixer's ``q_temp`` (queries keep their size at every
position), a router's ``identity`` (no identity experts), a routed
feed-forward's ``shared`` (no shared expert), ``mlp`` null (a layer without
feed-forward).
"""
from __future__ import annotations

from dataclasses import dataclass

from .base import ConfigError, KeyReader


@dataclass(frozen=True)
class QueryTemperature:
    coef: float
    every: int


@dataclass(frozen=True)
class ZuzenexAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: QueryTemperature | None


@dataclass(frozen=True)
class ZuzenexLightning:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]


@dataclass(frozen=True)
class ZuzenexFeedForward:
    kind: str              # "dense" or "moe"
    ff: int                # of the dense layer, or of one expert
    experts: int = 0
    identity: int = 0
    top: int = 0
    shared_ff: int = 0     # 0: no shared expert


@dataclass(frozen=True)
class ZuzenexLayer:
    mixer: ZuzenexAttention | ZuzenexLightning
    feed_forward: ZuzenexFeedForward | None


def _attention(m: KeyReader) -> ZuzenexAttention:
    temp = m.mapping("q_temp", None)
    if temp is not None:
        r = KeyReader(temp, m.source + ".q_temp")
        temp = QueryTemperature(r.number("coef", positive=False), r.integer("every"))
    a = ZuzenexAttention(heads=m.integer("heads"), kv_heads=m.integer("kv_heads"), dim=m.integer("dim"), vdim=m.integer("vdim"),
                         scale=m.number("scale", positive=False), q_temp=temp)
    if a.heads % a.kv_heads:
        raise ConfigError(f"{m.source}: {a.heads} heads do not divide into {a.kv_heads} kv_heads")
    return a


def _lightning(m: KeyReader) -> ZuzenexLightning:
    heads = m.integer("heads")
    decay = m.raw.get("decay")
    if decay is None:
        raise ConfigError(f"{m.source}: required key 'decay' is missing")
    if not isinstance(decay, list) or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
        raise ConfigError(f"{m.source}: 'decay' must be a list of numbers, got {decay!r}")
    if len(decay) != heads:
        raise ConfigError(f"{m.source}: 'decay' has {len(decay)} numbers for {heads} heads")
    if not all(0.0 <= d <= 1.0 for d in decay):
        raise ConfigError(f"{m.source}: a decay lies between 0 and 1, got {decay!r}")
    return ZuzenexLightning(heads=heads, dim=m.integer("dim"), vdim=m.integer("vdim"), decay=tuple(float(d) for d in decay))


def _feed_forward(f: KeyReader) -> ZuzenexFeedForward:
    kind = f.string("kind")
    if kind == "dense":
        return ZuzenexFeedForward("dense", f.integer("ff"))
    if kind != "moe":
        raise ConfigError(f"{f.source}: unknown kind {kind!r} (known: 'dense', 'moe')")
    router = KeyReader(f.mapping("router"), f.source + ".router")
    shared = f.mapping("shared", None)
    ff = ZuzenexFeedForward("moe", KeyReader(f.mapping("expert"), f.source + ".expert").integer("ff"),
                            experts=router.integer("experts"), identity=router.integer("identity", 0, minimum=0),
                            top=router.integer("top"),
                            shared_ff=KeyReader(shared, f.source + ".shared").integer("ff") if shared is not None else 0)
    if ff.top > ff.experts + ff.identity:
        raise ConfigError(f"{router.source}: top {ff.top} of {ff.experts} experts and {ff.identity} identity experts")
    return ff


@dataclass(frozen=True)
class ZuzenexConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    loop: tuple[int, int, int] | None  # (start, stop, times)
    layers: tuple[ZuzenexLayer, ...]
    raw: dict

    def run_order(self) -> list[int]:
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        start, stop, times = self.loop
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    @staticmethod
    def from_dict(raw: dict, source: str = "config.json") -> "ZuzenexConfig":
        r = KeyReader(raw, source)
        norm = KeyReader(r.mapping("norm"), source + ": norm")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError(f"{source}: 'layers' must be a non-empty list")
        readers = {"attention": _attention, "lightning": _lightning}
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
            ff = None
            if entry.get("mlp") is not None:
                ff = _feed_forward(KeyReader(e.mapping("mlp"), where + ".mlp"))
            layers.append(ZuzenexLayer(mixer, ff))
        loop = None
        raw_loop = r.mapping("loop", None)
        if raw_loop is not None:
            lp = KeyReader(raw_loop, source + ": loop")
            loop = (lp.integer("start", minimum=0), lp.integer("stop", minimum=0), lp.integer("times", minimum=0))
            if not loop[0] <= loop[1] <= len(layers):
                raise ConfigError(f"{source}: loop {loop[0]}..{loop[1]} does not lie within the {len(layers)} layers")
        return ZuzenexConfig(architecture=r.string("architecture"), vocab=r.integer("vocab"), width=r.integer("width"),
                             norm_eps=norm.number("eps"), loop=loop, layers=tuple(layers), raw=dict(raw))
