"""Configuration of the Nolapel decoder, read from its config.json.

    {"architecture": "Nolapel", "vocab": V, "width": W, "norm": {"eps": e},
     "embedding": {"bigram": {"buckets": n, "mul_prev": a, "mul_cur": b}}, "logit_softcap": c,
     "layers": [{"type": "attention" | "parallel" | "mamba2", "mixer": {...}, "mlp": {...} | null}, ...],
     "loop": {"start": a, "stop": b, "times": n}}

attention mixer: heads, kv_heads, dim, vdim (equal to dim: the values are keys), conv (taps), scale, mask {size},
                 q_temp {coef, every}.
parallel mixer: {"left": {heads, kv_heads, dim, vdim, scale, rot {dims, base}}, "left_scale": a,
                 "right": {heads, dim}, "right_scale": b}
mamba2 mixer: heads, vdim, state, groups, norm_groups, conv (taps).
mlp: {"kind": "moe", "router": {"experts": E, "top": k}, "expert": {"ff": F}, "shared": {"ff": S}}.
Every size and constant comes from the file.  What may be absent: `mlp` (no feed-forward), `loop` (every layer runs once),
`embedding` or its `bigram` (the token's row alone), `logit_softcap` (no cap), `mask` (every earlier position is seen),
`q_temp` (no temperature), `rot` (no rotation), `mlp.shared` (no shared expert), and the two scales of the parallel
mixer (1).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .base import ConfigError, KeyReader
from .zekivik import Loop, Rotation, _obj, _rotation

ATTENTION = "attention"
PARALLEL = "parallel"
MAMBA2 = "mamba2"


@dataclass(frozen=True)
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class BiasedAttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    conv: int
    scale: float
    window: int                              # 0: every earlier position is seen
    temperature: tuple[float, float] | None  # (coef, every)


@dataclass(frozen=True)
class SinkAttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotation                            # dims 0: no rotation


@dataclass(frozen=True)
class ParallelSizes:
    left: SinkAttentionSizes
    left_scale: float
    right_heads: int
    right_dim: int
    right_scale: float


@dataclass(frozen=True)
class Mamba2Sizes:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int


@dataclass(frozen=True)
class MoeSizes:
    experts: int
    top: int
    ff: int
    shared_ff: int                           # 0: no shared expert


@dataclass(frozen=True)
class NolapelLayer:
    type: str
    mixer: Any                               # BiasedAttentionSizes | ParallelSizes | Mamba2Sizes
    mlp: MoeSizes | None


@dataclass(frozen=True)
class NolapelConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    bigram: Bigram | None
    layers: tuple[NolapelLayer, ...]
    loop: Loop | None
    logit_softcap: float                     # 0: no cap

    @staticmethod
    def from_dict(raw: dict[str, Any]) -> "NolapelConfig":
        r = KeyReader(raw)
        norm = _obj(r, "norm", "config.json")
        entries = r.array("layers", item=lambda e: isinstance(e, dict))
        if not entries:
            raise ConfigError("config.json: 'layers' is empty")
        layers = tuple(_layer(e, f"config.json: layers[{i}]") for i, e in enumerate(entries))
        loop = None
        if r.has("loop"):
            lp = _obj(r, "loop", "config.json")
            loop = Loop(lp.integer("start", minimum=0), lp.integer("stop", minimum=0), lp.integer("times", minimum=1))
            if not loop.start <= loop.stop <= len(layers):
                raise ConfigError(f"config.json: loop {loop.start}..{loop.stop} does not fit {len(layers)} layers")
        bigram = None
        if r.has("embedding"):
            er = _obj(r, "embedding", "config.json")
            if er.has("bigram"):
                br = _obj(er, "bigram", "config.json: embedding")
                bigram = Bigram(br.integer("buckets", minimum=1), br.integer("mul_prev", minimum=0), br.integer("mul_cur", minimum=0))
        cap = r.number("logit_softcap", default=0.0)
        if cap < 0:
            raise ConfigError(f"config.json: 'logit_softcap' must not be negative, got {cap}")
        return NolapelConfig(
            architecture=r.string("architecture"), vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
            eps=norm.number("eps"), bigram=bigram, layers=layers, loop=loop, logit_softcap=cap)

    def runs(self) -> list[tuple[int, int | None]]:
        """(layer, number of the pass it opens or None) in running order: the layers before the loop once, the looped
        range `times` times as a whole, the rest once."""
        n = len(self.layers)
        if self.loop is None or self.loop.stop == self.loop.start:
            return [(i, None) for i in range(n)]
        a, b, times = self.loop.start, self.loop.stop, self.loop.times
        order: list[tuple[int, int | None]] = [(i, None) for i in range(a)]
        for t in range(times):
            order += [(i, t if i == a else None) for i in range(a, b)]
        return order + [(i, None) for i in range(b, n)]


def _heads(mr: KeyReader, where: str) -> tuple[int, int]:
    heads, kv = mr.integer("heads", minimum=1), mr.integer("kv_heads", minimum=1)
    if heads % kv:
        raise ConfigError(f"{where}: {heads} heads do not divide into {kv} kv_heads")
    return heads, kv


def _layer(e: dict, where: str) -> NolapelLayer:
    lr = KeyReader(e, where)
    kind = lr.string("type")
    mr = _obj(lr, "mixer", where)
    mixer: Any
    if kind == ATTENTION:
        heads, kv = _heads(mr, where)
        temperature = None
        if mr.has("q_temp"):
            tr = _obj(mr, "q_temp", where)
            temperature = (tr.number("coef"), tr.number("every"))
            if not temperature[1] > 0:
                raise ConfigError(f"{where}: q_temp.every must be positive, got {temperature[1]}")
        mixer = BiasedAttentionSizes(
            heads=heads, kv_heads=kv, dim=mr.integer("dim", minimum=1), conv=mr.integer("conv", minimum=1), scale=mr.number("scale"),
            window=_obj(mr, "mask", where).integer("size", minimum=1) if mr.has("mask") else 0, temperature=temperature)
        if mr.integer("vdim", default=mixer.dim) != mixer.dim:
            raise ConfigError(f"{where}: the values are keys, so vdim must be dim ({mixer.dim}), got {mr.raw['vdim']}")
    elif kind == PARALLEL:
        ar, rr = _obj(mr, "left", where), _obj(mr, "right", where)
        heads, kv = _heads(ar, f"{where}: left")
        rot = _rotation(ar, where) if ar.has("rot") else Rotation(0, 10000.0)
        left = SinkAttentionSizes(heads=heads, kv_heads=kv, dim=ar.integer("dim", minimum=1), vdim=ar.integer("vdim", minimum=1),
                                  scale=ar.number("scale"), rot=rot)
        if rot.dims > left.dim:
            raise ConfigError(f"{where}: rot.dims {rot.dims} is more than dim {left.dim}")
        mixer = ParallelSizes(left=left, left_scale=mr.number("left_scale", default=1.0),
                              right_heads=rr.integer("heads", minimum=1), right_dim=rr.integer("dim", minimum=1),
                              right_scale=mr.number("right_scale", default=1.0))
    elif kind == MAMBA2:
        mixer = Mamba2Sizes(**{k: mr.integer(k, minimum=1) for k in ("heads", "vdim", "state", "groups", "norm_groups", "conv")})
        if mixer.heads % mixer.groups:
            raise ConfigError(f"{where}: {mixer.heads} heads do not divide into {mixer.groups} groups")
        if (mixer.heads * mixer.vdim) % mixer.norm_groups:
            raise ConfigError(f"{where}: {mixer.heads} x {mixer.vdim} channels do not divide into {mixer.norm_groups} norm_groups")
    else:
        raise ConfigError(f"{where}: unknown layer type '{kind}' ({ATTENTION}, {MAMBA2}, {PARALLEL})")
    return NolapelLayer(kind, mixer, _mlp(lr, where))


def _mlp(lr: KeyReader, where: str) -> MoeSizes | None:
    if not lr.has("mlp"):
        return None
    fr = _obj(lr, "mlp", where)
    kind = fr.string("kind")
    if kind != "moe":
        raise ConfigError(f"{where}: unknown mlp kind '{kind}' (moe)")
    rr = _obj(fr, "router", where)
    m = MoeSizes(experts=rr.integer("experts", minimum=1), top=rr.integer("top", minimum=1),
                 ff=_obj(fr, "expert", where).integer("ff", minimum=1),
                 shared_ff=_obj(fr, "shared", where).integer("ff", minimum=1) if fr.has("shared") else 0)
    if m.top > m.experts:
        raise ConfigError(f"{where}: top {m.top} of {m.experts} experts")
    return m
