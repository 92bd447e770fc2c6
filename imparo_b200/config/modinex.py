"""Typed configuration of Modinex, read from its config.json keys.

A decoder-only design: the embedding row plus a learned vector per position; every sublayer has a norm before it and a norm
on its output (`norm.groups` equal stretches of the row, each by its own root mean square).  `layers` lists the layers in any
order; each names its mixer:

  "attention"  grouped-query attention with weighted RMS norms on each query and key head, half-split rotation over the
               first `rot.dims` dimensions, an explicit score scale, a mask that cuts the sequence into stretches of
               `mask.size` positions, and no softmax: a visible key weighs sigmoid(score + a number per head);
  "gla"        gated linear attention with a decay per key channel, sigmoid(z)^(1/`tau`), a per-head norm and a silu gate;

and its feed-forward (`mlp`): "dense" (up, tanh gelu, down, with biases), or null.  Every size and constant comes from
config.json, except the inner size of the two-step decay projection, which is the stored tensor's; an absent optional key
switches its mechanism off (no `mask`: all earlier positions; no `rot`: no rotation; `kv_heads` = heads; `vdim` = dim;
`norm.groups` 1; no `max_positions`: no position vectors).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple, Union

from .base import ConfigError, KeyReader

LAYER_TYPES = ("attention", "gla")
MLP_KINDS = ("dense",)


@dataclass(frozen=True)
class AttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: Optional[int]              # a position sees only its own stretch of this many; None: all before it
    rot_dims: int                     # 0: no rotation
    rot_base: float


@dataclass(frozen=True)
class GlaSizes:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: Optional[int]               # inner size of the decay's two-step projection where no stored tensor gives it


@dataclass(frozen=True)
class DenseSizes:
    ff: int


@dataclass(frozen=True)
class ModinexLayer:
    type: str
    mixer: Union[AttentionSizes, GlaSizes]
    mlp: Optional[DenseSizes]


@dataclass(frozen=True)
class ModinexConfig:
    vocab: int
    width: int
    eps: float
    groups: int
    max_positions: Optional[int]      # rows of the position table; None: the model has none
    layers: Tuple[ModinexLayer, ...]


def _sub(reader: KeyReader, key: str, required: bool = True) -> Optional[KeyReader]:
    v = reader.raw(key)
    if v is None:
        if required:
            raise ConfigError(f"{reader.where}: missing required key '{key}'")
        return None
    return KeyReader(v, f"{reader.where}: {key}")


def _attention(r: KeyReader) -> AttentionSizes:
    heads = r.integer("heads", minimum=1)
    kv = r.integer("kv_heads", default=heads, minimum=1)
    if heads % kv:
        raise ConfigError(f"{r.where}: kv_heads {kv} must divide heads {heads}")
    dim = r.integer("dim", minimum=1)
    rot = _sub(r, "rot", required=False)
    rot_dims, rot_base = 0, 10000.0
    if rot is not None:
        rot_dims, rot_base = rot.integer("dims", default=dim, minimum=0), rot.number("base")
        if rot_dims % 2 or rot_dims > dim:
            raise ConfigError(f"{rot.where}: dims {rot_dims} must be even and at most dim {dim}")
    mask = _sub(r, "mask", required=False)
    return AttentionSizes(heads=heads, kv_heads=kv, dim=dim, vdim=r.integer("vdim", default=dim, minimum=1), scale=r.number("scale"),
                          chunk=mask.integer("size", minimum=1) if mask is not None else None, rot_dims=rot_dims, rot_base=rot_base)


def _gla(r: KeyReader) -> GlaSizes:
    tau = r.number("tau")
    if not tau > 0.0:
        raise ConfigError(f"{r.where}: tau must be positive, found {tau}")
    return GlaSizes(heads=r.integer("heads", minimum=1), dim=r.integer("dim", minimum=1), vdim=r.integer("vdim", minimum=1), tau=tau,
                    rank=r.integer("rank", default=None, minimum=1))


_MIXERS = {"attention": _attention, "gla": _gla}


def _mlp(r: Optional[KeyReader]) -> Optional[DenseSizes]:
    if r is None:
        return None
    kind = r.raw("kind")
    if kind not in MLP_KINDS:
        raise ConfigError(f"{r.where}: unknown kind {kind!r}; known: {', '.join(MLP_KINDS)}")
    return DenseSizes(ff=r.integer("ff", minimum=1))


def parse_modinex_config(values: dict) -> ModinexConfig:
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
        layers.append(ModinexLayer(type=kind, mixer=_MIXERS[kind](_sub(lr, "mixer")), mlp=_mlp(_sub(lr, "mlp", required=False))))
    norm = _sub(r, "norm")
    width, groups = r.integer("width", minimum=1), norm.integer("groups", default=1, minimum=1)
    if width % groups:
        raise ConfigError(f"{norm.where}: groups {groups} must divide width {width}")
    return ModinexConfig(vocab=r.integer("vocab", minimum=1), width=width, eps=norm.number("eps"), groups=groups,
                         max_positions=r.integer("max_positions", default=None, minimum=1), layers=tuple(layers))
