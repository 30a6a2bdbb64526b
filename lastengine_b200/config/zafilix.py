"""Configuration of the Zafilix decoder, read from its config.json.

    {"architecture": "Zafilix", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
     "logit_scale": a, "logit_softcap": c,
     "layers": [{"type": "attention" | "latent_attention", "mixer": {...}, "mlp": {"kind": "dense", "ff": F} | null,
                 "weights_of": j}, ...]}

attention mixer: heads, kv_heads, dim, vdim, scale, rot {dims, base, scaling {factor}}, mask {size} (chunks of `size`
positions).
latent_attention mixer: heads, dim, rot_dim, vdim, kv_rank, scale, rot {dims, base, scaling {factor}}, mask {size} (a
window of `size` positions).
`weights_of`: the layer runs layer j's tensors (mixer, feed-forward and norms) with a memory of its own.
Every size and constant comes from the file.  What may be absent: `mlp` (no feed-forward), `weights_of` (tensors of
its own), `mask` (plain causal attention), `rot` (no rotation), `rot.scaling` (factor 1), `embedding` (scale 1),
`logit_scale` (1) and `logit_softcap` (no cap).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .base import ConfigError, KeyReader
from .tevilix import ScaledRotation
from .zekivik import _obj

ATTENTION = "attention"
LATENT = "latent_attention"


@dataclass(frozen=True)
class ChunkedAttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: ScaledRotation
    chunk: int             # 0: every earlier position is seen


@dataclass(frozen=True)
class LatentSizes:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: ScaledRotation
    window: int            # 0: every earlier position is seen


@dataclass(frozen=True)
class ZafilixLayer:
    type: str
    mixer: Any             # ChunkedAttentionSizes | LatentSizes
    ff: int | None         # width of the dense feed-forward, None: the layer has none
    owner: int             # the layer whose tensors this one runs (itself, unless it borrows another's)


@dataclass(frozen=True)
class ZafilixConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_scale: float
    logit_softcap: float   # 0: no cap
    layers: tuple[ZafilixLayer, ...]

    @staticmethod
    def from_dict(raw: dict[str, Any]) -> "ZafilixConfig":
        r = KeyReader(raw)
        norm = _obj(r, "norm", "config.json")
        entries = r.array("layers", item=lambda e: isinstance(e, dict))
        if not entries:
            raise ConfigError("config.json: 'layers' is empty")
        own = [_layer(e, i) for i, e in enumerate(entries)]
        layers = []
        for i, (kind, mixer, ff, _) in enumerate(own):
            j = _owner(own, i)
            if own[j][:3] != (kind, mixer, ff):
                raise ConfigError(f"config.json: layers[{i}] runs the weights of layer {j} and must have its type and sizes")
            layers.append(ZafilixLayer(kind, mixer, ff, j))
        cap = r.number("logit_softcap", default=0.0)
        if cap < 0:
            raise ConfigError(f"config.json: 'logit_softcap' must not be negative, got {cap}")
        return ZafilixConfig(
            architecture=r.string("architecture"), vocab=r.integer("vocab", minimum=1),
            width=r.integer("width", minimum=1), eps=norm.number("eps"),
            embedding_scale=_obj(r, "embedding", "config.json").number("scale", default=1.0) if r.has("embedding") else 1.0,
            logit_scale=r.number("logit_scale", default=1.0), logit_softcap=cap, layers=tuple(layers))

    def owners(self) -> list[int]:
        """The layers that have tensors of their own, in order."""
        return [i for i, lay in enumerate(self.layers) if lay.owner == i]


def _owner(own: list, i: int) -> int:
    """Follows `weights_of` to the layer that has the tensors."""
    seen = [i]
    while own[seen[-1]][3] is not None:
        j = own[seen[-1]][3]
        if j >= len(own):
            raise ConfigError(f"config.json: layers[{seen[-1]}]: weights_of {j} of {len(own)} layers")
        if j in seen:
            raise ConfigError(f"config.json: layers[{i}]: weights_of goes round in a circle ({' -> '.join(map(str, seen + [j]))})")
        seen.append(j)
    return seen[-1]


def _layer(e: dict, i: int) -> tuple:
    """(type, mixer sizes, feed-forward width or None, weights_of or None)."""
    where = f"config.json: layers[{i}]"
    lr = KeyReader(e, where)
    kind = lr.string("type")
    mr = _obj(lr, "mixer", where)
    reach = _obj(mr, "mask", where).integer("size", minimum=1) if mr.has("mask") else 0
    rot = _rotation(mr, where)
    if kind == ATTENTION:
        mixer = ChunkedAttentionSizes(
            heads=mr.integer("heads", minimum=1), kv_heads=mr.integer("kv_heads", minimum=1), dim=mr.integer("dim", minimum=1),
            vdim=mr.integer("vdim", minimum=1), scale=mr.number("scale"), rot=rot, chunk=reach)
        if mixer.heads % mixer.kv_heads:
            raise ConfigError(f"{where}: {mixer.heads} heads do not divide into {mixer.kv_heads} kv_heads")
        if rot.dims > mixer.dim:
            raise ConfigError(f"{where}: rot.dims {rot.dims} is more than dim {mixer.dim}")
    elif kind == LATENT:
        mixer = LatentSizes(
            heads=mr.integer("heads", minimum=1), dim=mr.integer("dim", minimum=1), rot_dim=mr.integer("rot_dim", minimum=0),
            vdim=mr.integer("vdim", minimum=1), kv_rank=mr.integer("kv_rank", minimum=1), scale=mr.number("scale"), rot=rot,
            window=reach)
        if rot.dims > mixer.rot_dim:
            raise ConfigError(f"{where}: rot.dims {rot.dims} is more than rot_dim {mixer.rot_dim}")
    else:
        raise ConfigError(f"{where}: unknown layer type '{kind}' ({ATTENTION}, {LATENT})")
    ff = None
    if lr.has("mlp"):
        fr = _obj(lr, "mlp", where)
        fk = fr.string("kind")
        if fk != "dense":
            raise ConfigError(f"{where}: unknown mlp kind '{fk}' (dense)")
        ff = fr.integer("ff", minimum=1)
    return kind, mixer, ff, lr.integer("weights_of", minimum=0) if lr.has("weights_of") else None


def _rotation(mr: KeyReader, where: str) -> ScaledRotation:
    if not mr.has("rot"):
        return ScaledRotation(0, 10000.0, 1.0)
    rr = _obj(mr, "rot", where)
    dims = rr.integer("dims", minimum=0)
    if dims % 2:
        raise ConfigError(f"{where}: rot.dims must be even, got {dims}")
    factor = _obj(rr, "scaling", where).number("factor", default=1.0) if rr.has("scaling") else 1.0
    if not factor > 0:
        raise ConfigError(f"{where}: rot.scaling.factor must be positive, got {factor}")
    return ScaledRotation(dims, rr.number("base"), factor)
