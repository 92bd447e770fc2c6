"""Typed configuration of Zinunex, read from its config.json keys.

A decoder-only design: pre-norm layers (RMS norms), each a mixer, a routed feed-forward (or none) and a token input of its own.
`layers` lists the layers in any order; each names its mixer:

  "latent_attention"  queries straight from the input, per head [dim plain | rot_dim rotated]; keys and values from one
                      normed latent of kv_rank per token plus one rotated key part of rot_dim that all heads share (the
                      cache keeps those two); rotation of neighbouring pairs, optionally with scaled frequencies and a magnitude
                      (`rot.scaling`: factor, original, fast, slow); a sliding window (`mask.size`); softmax.  `kv_from`: the
                      layer makes no latent and reads the cache of that earlier layer;
  "attention"         grouped queries, values are the keys before the rotation, half-split rotation of the first `rot.dims`
                      dimensions, frequencies optionally divided by `rot.scaling.factor`; causal softmax with a learned number
                      per head in the denominator;

and its feed-forward (`mlp`): "moe" (sigmoid router with a correction per expert that only the choice sees; experts in equal
groups of neighbours, a group's score the sum of its two largest choice scores, only the best `groups.keep` groups' experts may be
chosen; `top` experts, weights times `router.scale`; squared-relu experts without a gate; an optional shared expert with a factor per
token), or null.  Every size and constant below comes from config.json; an absent optional key switches its mechanism off (no
`mask`: all earlier positions; no `rot`: no rotation; no `scaling`: plain frequencies; no `groups`: every expert may be chosen; no
`shared`: no shared expert; no `token_side`: no token input per layer).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple, Union

from .base import ConfigError, KeyReader

LAYER_TYPES = ("latent_attention", "attention")


@dataclass(frozen=True)
class BlendedScaling:
    """Frequencies between the plain ones and those divided by `factor`, by how often a pair turns over `original` positions."""
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class LatentSizes:
    heads: int
    dim: int                          # unrotated query/key dimensions per head
    rot_dim: int                      # rotated dimensions per head (the key's are shared by all heads); 0: none
    vdim: int
    kv_rank: int
    scale: float
    window: Optional[int]
    kv_from: Optional[int]            # the layer whose cache this one reads; None: its own
    rot_dims: int                     # how many of the rot_dim dimensions turn (the first ones)
    rot_base: float
    rot_scaling: Optional[BlendedScaling]


@dataclass(frozen=True)
class AttentionSizes:
    heads: int
    kv_heads: int
    dim: int                          # query/key size and, values being keys, value size
    scale: float
    rot_dims: int
    rot_base: float
    rot_factor: float                 # divides every frequency (1: plain)


@dataclass(frozen=True)
class MoeSizes:
    experts: int
    top: int
    groups: int                       # 1: no groups
    keep: int
    scale: float
    ff: int                           # per expert
    shared_ff: Optional[int]


@dataclass(frozen=True)
class ZinunexLayer:
    type: str
    mixer: Union[LatentSizes, AttentionSizes]
    mlp: Optional[MoeSizes]


@dataclass(frozen=True)
class ZinunexConfig:
    vocab: int
    width: int
    eps: float
    side_dim: Optional[int]           # entries of the token input per layer; None: the layers have none
    layers: Tuple[ZinunexLayer, ...]


def _sub(reader: KeyReader, key: str, required: bool = True) -> Optional[KeyReader]:
    v = reader.raw(key)
    if v is None:
        if required:
            raise ConfigError(f"{reader.where}: missing required key '{key}'")
        return None
    return KeyReader(v, f"{reader.where}: {key}")


def _rot_dims(rot: KeyReader, most: int, of: str) -> int:
    dims = rot.integer("dims", default=most, minimum=0)
    if dims % 2 or dims > most:
        raise ConfigError(f"{rot.where}: dims {dims} must be even and at most {of} {most}")
    return dims


def _positive(r: KeyReader, key: str) -> float:
    v = r.number(key)
    if not v > 0.0:
        raise ConfigError(f"{r.where}: {key} must be positive, found {v}")
    return v


def _latent(r: KeyReader) -> LatentSizes:
    rot_dim = r.integer("rot_dim", default=0, minimum=0)
    rot = _sub(r, "rot", required=False)
    rot_dims, rot_base, scaling = 0, 10000.0, None
    if rot is not None and rot_dim:
        rot_dims, rot_base = _rot_dims(rot, rot_dim, "rot_dim"), _positive(rot, "base")
        sc = _sub(rot, "scaling", required=False)
        if sc is not None:
            scaling = BlendedScaling(*(_positive(sc, k) for k in ("factor", "original", "fast", "slow")))
    mask = _sub(r, "mask", required=False)
    return LatentSizes(heads=r.integer("heads", minimum=1), dim=r.integer("dim", minimum=1), rot_dim=rot_dim,
                       vdim=r.integer("vdim", minimum=1), kv_rank=r.integer("kv_rank", minimum=1), scale=r.number("scale"),
                       window=mask.integer("size", minimum=1) if mask is not None else None,
                       kv_from=r.integer("kv_from", default=None, minimum=0), rot_dims=rot_dims, rot_base=rot_base, rot_scaling=scaling)


def _attention(r: KeyReader) -> AttentionSizes:
    heads = r.integer("heads", minimum=1)
    kv = r.integer("kv_heads", default=heads, minimum=1)
    if heads % kv:
        raise ConfigError(f"{r.where}: kv_heads {kv} must divide heads {heads}")
    dim = r.integer("dim", minimum=1)
    vdim = r.integer("vdim", default=dim, minimum=1)
    if vdim != dim:
        raise ConfigError(f"{r.where}: the values are the keys, so vdim {vdim} must equal dim {dim}")
    rot = _sub(r, "rot", required=False)
    rot_dims, rot_base, factor = 0, 10000.0, 1.0
    if rot is not None:
        rot_dims, rot_base = _rot_dims(rot, dim, "dim"), _positive(rot, "base")
        sc = _sub(rot, "scaling", required=False)
        if sc is not None:
            factor = _positive(sc, "factor")
    return AttentionSizes(heads=heads, kv_heads=kv, dim=dim, scale=r.number("scale"), rot_dims=rot_dims, rot_base=rot_base, rot_factor=factor)


_MIXERS = {"latent_attention": _latent, "attention": _attention}


def _moe(r: Optional[KeyReader]) -> Optional[MoeSizes]:
    if r is None:
        return None
    if r.raw("kind") != "moe":
        raise ConfigError(f"{r.where}: unknown kind {r.raw('kind')!r}; known: moe")
    router = _sub(r, "router")
    experts, top = router.integer("experts", minimum=1), router.integer("top", minimum=1)
    if top > experts:
        raise ConfigError(f"{router.where}: top {top} exceeds experts {experts}")
    groups = _sub(router, "groups", required=False)
    count, keep = 1, 1
    if groups is not None:
        count = groups.integer("count", minimum=1)
        keep = groups.integer("keep", default=count, minimum=1)
        if experts % count or keep > count:
            raise ConfigError(f"{groups.where}: count {count} must divide experts {experts} and keep {keep} must not exceed it")
        if keep * (experts // count) < top:
            raise ConfigError(f"{groups.where}: {keep} groups of {experts // count} experts cannot give top {top}")
    shared = _sub(r, "shared", required=False)
    return MoeSizes(experts=experts, top=top, groups=count, keep=keep, scale=router.number("scale", default=1.0),
                    ff=_sub(r, "expert").integer("ff", minimum=1),
                    shared_ff=shared.integer("ff", minimum=1) if shared is not None else None)


def _check_sources(layers) -> None:
    for i, L in enumerate(layers):
        j = getattr(L.mixer, "kv_from", None)
        if j is None:
            continue
        where = f"config.json: layers[{i}]: kv_from {j}"
        if j >= i or layers[j].type != "latent_attention":
            raise ConfigError(f"{where} must name an earlier latent_attention layer")
        src = layers[j].mixer
        if src.kv_from is not None:
            raise ConfigError(f"{where} names a layer that makes no latent of its own")
        same = ("kv_rank", "rot_dim", "rot_dims", "rot_base", "rot_scaling")
        if any(getattr(src, k) != getattr(L.mixer, k) for k in same):
            raise ConfigError(f"{where}: both layers need the same kv_rank, rot_dim and rotation")


def parse_zinunex_config(values: dict) -> ZinunexConfig:
    r = KeyReader(values)
    layers_raw = r.raw("layers")
    if not isinstance(layers_raw, list) or not layers_raw:
        raise ConfigError("config.json: key 'layers' must be a non-empty list")
    layers = []
    for i, entry in enumerate(layers_raw):
        lr = KeyReader(entry, f"config.json: layers[{i}]")
        kind = lr.raw("type")
        if kind not in LAYER_TYPES:
            raise ConfigError(f"{lr.where}: unknown type {kind!r}; known: {', '.join(LAYER_TYPES)}")
        layers.append(ZinunexLayer(type=kind, mixer=_MIXERS[kind](_sub(lr, "mixer")), mlp=_moe(_sub(lr, "mlp", required=False))))
    _check_sources(layers)
    side = _sub(r, "token_side", required=False)
    return ZinunexConfig(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1), eps=_sub(r, "norm").number("eps"),
                         side_dim=side.integer("dim", minimum=1) if side is not None else None, layers=tuple(layers))
