"""Typed view of a Tupunex ``config.json``.

Tupunex is a decoder-only model with a nested configuration: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``,
``streams`` (residual streams side by side), an optional ``loop`` (``start``, ``stop``, ``times``: layers start .. stop-1 run that
many times in a row) and a list ``layers`` whose entries give the layer's ``type`` (``attention``: differential attention inside
a sliding window behind a short convolution; ``latent_attention``), the mixer's sizes and constants (``mixer``) and its
feed-forward (``mlp``: ``kind`` ``dense``, or null for none).  Every size and constant is read from there; what an entry does
not mention is off; a layer type or feed-forward kind that is not understood is refused by name.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple, Union

from .dosovik_config import _get
from .model_config import ConfigError
from .tutezen_config import Loop


@dataclass(frozen=True)
class DifferentialAttentionSizes:
    heads: int
    kv_heads: int
    dim: int                     # size of one map of a query / key head (a head has two)
    vdim: int
    scale: float
    diff: float                  # the constant part of the second map's weight
    conv: int                    # taps of the convolution on q, k and v (0: none)
    softcap: Optional[float]     # score <- softcap * tanh(score / softcap)
    window: Optional[int]        # mask.size: a position sees itself and the window - 1 before it (None: all)


@dataclass(frozen=True)
class SharedLatentSizes:
    heads: int
    dim: int                     # unrotated query/key dimensions of a head
    rot_dim: int                 # rotated query/key dimensions of a head (the key part is shared by all heads)
    vdim: int
    kv_rank: int
    scale: float
    rot_dims: int                # how many leading dimensions of the rotated part turn (0: none)
    rot_base: float


@dataclass(frozen=True)
class DenseFF:
    ff: int


@dataclass(frozen=True)
class TupunexLayer:
    type: str
    mixer: Union[DifferentialAttentionSizes, SharedLatentSizes]
    mlp: Optional[DenseFF]


def _positive(v, where: str):
    if v <= 0:
        raise ConfigError(f"config.json {where} must be positive, got {v}")
    return v


def _differential(m: dict, where: str) -> DifferentialAttentionSizes:
    pos = lambda key: _positive(_get(m, key, int, where), where + key)  # noqa: E731
    heads, kv_heads = pos("heads"), pos("kv_heads")
    if heads % kv_heads:
        raise ConfigError(f"config.json {where}heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    mask = _get(m, "mask", dict, where, required=False)
    conv = _get(m, "conv", int, where, default=0, required=False)
    if conv < 0:
        raise ConfigError(f"config.json {where}conv must not be negative, got {conv}")
    cap = _get(m, "softcap", float, where, required=False)
    return DifferentialAttentionSizes(
        heads=heads, kv_heads=kv_heads, dim=pos("dim"), vdim=pos("vdim"), scale=_get(m, "scale", float, where),
        diff=_get(m, "diff", float, where), conv=conv, softcap=_positive(cap, where + "softcap") if cap is not None else None,
        window=_positive(_get(mask, "size", int, where + "mask."), where + "mask.size") if mask is not None else None)


def _latent(m: dict, where: str) -> SharedLatentSizes:
    pos = lambda key: _positive(_get(m, key, int, where), where + key)  # noqa: E731
    rot_dim = pos("rot_dim")
    rot = _get(m, "rot", dict, where, required=False)
    rot_dims = _get(rot, "dims", int, where + "rot.") if rot is not None else 0
    if rot_dims < 0 or rot_dims % 2 or rot_dims > rot_dim:
        raise ConfigError(f"config.json {where}rot.dims ({rot_dims}) must be even and at most rot_dim ({rot_dim})")
    return SharedLatentSizes(heads=pos("heads"), dim=pos("dim"), rot_dim=rot_dim, vdim=pos("vdim"), kv_rank=pos("kv_rank"),
                             scale=_get(m, "scale", float, where), rot_dims=rot_dims,
                             rot_base=_positive(_get(rot, "base", float, where + "rot."), where + "rot.base") if rot_dims else 1.0)


def _mlp(mlp, where: str) -> Optional[DenseFF]:
    if mlp is None:
        return None
    kind = _get(mlp, "kind", str, where)
    if kind != "dense":
        raise ConfigError(f"config.json {where}kind {kind!r} is not known (known: 'dense')")
    return DenseFF(ff=_positive(_get(mlp, "ff", int, where), where + "ff"))


@dataclass(frozen=True)
class TupunexConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    streams: int
    loop: Optional[Loop]
    layers: Tuple[TupunexLayer, ...]

    architecture = "Tupunex"

    @staticmethod
    def from_dict(d: dict) -> "TupunexConfig":
        if not isinstance(d.get("layers"), list) or not d["layers"]:
            raise ConfigError("config.json needs a non-empty list 'layers'")
        layers = []
        for i, ly in enumerate(d["layers"]):
            where = f"layers[{i}]."
            kind = _get(ly, "type", str, where)
            m, mw = _get(ly, "mixer", dict, where), where + "mixer."
            if kind == "attention":
                mixer = _differential(m, mw)
            elif kind == "latent_attention":
                mixer = _latent(m, mw)
            else:
                raise ConfigError(f"config.json {where}type {kind!r} is not a mixer of this design "
                                  f"(known: 'attention', 'latent_attention')")
            layers.append(TupunexLayer(kind, mixer, _mlp(ly.get("mlp"), where + "mlp.")))
        loop = _get(d, "loop", dict, "", required=False)
        if loop is not None:
            loop = Loop(_get(loop, "start", int, "loop."), _get(loop, "stop", int, "loop."), _get(loop, "times", int, "loop."))
            if not (0 <= loop.start < loop.stop <= len(layers)) or loop.times < 1:
                raise ConfigError(f"config.json loop {loop} does not fit {len(layers)} layers")
        emb = _get(d, "embedding", dict, "", required=False)
        return TupunexConfig(
            vocab=_positive(_get(d, "vocab", int, ""), "vocab"), width=_positive(_get(d, "width", int, ""), "width"),
            eps=_get(_get(d, "norm", dict, ""), "eps", float, "norm."),
            embedding_scale=_get(emb, "scale", float, "embedding.", default=1.0, required=False) if emb is not None else 1.0,
            streams=_positive(_get(d, "streams", int, "", default=1, required=False), "streams"), loop=loop, layers=tuple(layers))
