"""Typed view of a Kavotar ``config.json``.

Kavotar is a decoder-only model with a nested configuration: ``vocab``, ``width``, ``norm.eps``, ``logit_softcap`` and a list
``layers`` whose entries give the layer's ``type`` (``mlstm``: a matrix memory with exponential gates; ``parallel``: attention
with weights mixed across heads and a decaying matrix state with a bonus, side by side, under ``mixer.left`` and
``mixer.right``), the mixer's sizes and constants (``mixer``) and its feed-forward (``mlp``: ``kind`` ``moe``, or null for
none).  Every size and constant is read from there; what a layer's entry does not mention is off; a layer type or
feed-forward kind that is not understood is refused by name.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple, Union

from .dosovik_config import _get
from .model_config import ConfigError


@dataclass(frozen=True)
class MemorySizes:               # type "mlstm"
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class TalkingAttention:          # the left side of type "parallel"
    heads: int
    kv_heads: int
    dim: int                     # size of a query / key head
    vdim: int                    # size of a value head
    scale: float
    chunk: Optional[int]         # mask.size: a position sees its own chunk only (None: everything before it)
    rot_dims: int                # 0: no rotation
    rot_base: float


@dataclass(frozen=True)
class BonusSizes:                # the right side of type "parallel"
    heads: int
    dim: int


@dataclass(frozen=True)
class SideBySideSizes:
    left: TalkingAttention
    right: BonusSizes


@dataclass(frozen=True)
class ExpertsFF:
    ff: int
    experts: int
    top: int
    groups: Optional[Tuple[int, int]]   # (count, keep)


@dataclass(frozen=True)
class KavotarLayer:
    type: str
    mixer: Union[MemorySizes, SideBySideSizes]
    mlp: Optional[ExpertsFF]


def _positive(v, where: str):
    if v <= 0:
        raise ConfigError(f"config.json {where} must be positive, got {v}")
    return v


def _pos(d: dict, key: str, where: str) -> int:
    return _positive(_get(d, key, int, where), where + key)


def _attention(m: dict, where: str) -> TalkingAttention:
    heads, kv_heads, dim = _pos(m, "heads", where), _pos(m, "kv_heads", where), _pos(m, "dim", where)
    if heads % kv_heads:
        raise ConfigError(f"config.json {where}heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    mask, rot = _get(m, "mask", dict, where, required=False), _get(m, "rot", dict, where, required=False)
    rot_dims = _get(rot, "dims", int, where + "rot.") if rot is not None else 0
    if rot_dims < 0 or rot_dims % 2 or rot_dims > dim:
        raise ConfigError(f"config.json {where}rot.dims ({rot_dims}) must be even and at most dim ({dim})")
    return TalkingAttention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=_pos(m, "vdim", where), scale=_get(m, "scale", float, where),
                            chunk=_pos(mask, "size", where + "mask.") if mask is not None else None, rot_dims=rot_dims,
                            rot_base=_positive(_get(rot, "base", float, where + "rot."), where + "rot.base") if rot_dims else 1.0)


def _mlp(mlp, where: str) -> Optional[ExpertsFF]:
    if mlp is None:
        return None
    kind = _get(mlp, "kind", str, where)
    if kind != "moe":
        raise ConfigError(f"config.json {where}kind {kind!r} is not known (known: 'moe')")
    e, r, rw = _get(mlp, "expert", dict, where), _get(mlp, "router", dict, where), where + "router."
    experts, top = _pos(r, "experts", rw), _pos(r, "top", rw)
    if top > experts:
        raise ConfigError(f"config.json {rw}top ({top}) must not exceed {rw}experts ({experts})")
    g, groups = _get(r, "groups", dict, rw, required=False), None
    if g is not None:
        groups = (_pos(g, "count", rw + "groups."), _pos(g, "keep", rw + "groups."))
        if experts % groups[0] or groups[1] > groups[0] or groups[1] * (experts // groups[0]) < top:
            raise ConfigError(f"config.json {rw}groups: {experts} experts in {groups[0]} equal groups of which {groups[1]} are kept "
                              f"cannot give {top}")
    return ExpertsFF(ff=_pos(e, "ff", where + "expert."), experts=experts, top=top, groups=groups)


@dataclass(frozen=True)
class KavotarConfig:
    vocab: int
    width: int
    eps: float
    logit_softcap: Optional[float]
    layers: Tuple[KavotarLayer, ...]

    architecture = "Kavotar"

    @staticmethod
    def from_dict(d: dict) -> "KavotarConfig":
        if not isinstance(d.get("layers"), list) or not d["layers"]:
            raise ConfigError("config.json needs a non-empty list 'layers'")
        layers = []
        for i, ly in enumerate(d["layers"]):
            where = f"layers[{i}]."
            kind = _get(ly, "type", str, where)
            m, mw = _get(ly, "mixer", dict, where), where + "mixer."
            if kind == "mlstm":
                mixer = MemorySizes(heads=_pos(m, "heads", mw), dim=_pos(m, "dim", mw), vdim=_pos(m, "vdim", mw),
                                    gate_cap=_positive(_get(m, "gate_cap", float, mw), mw + "gate_cap"))
            elif kind == "parallel":
                right = _get(m, "right", dict, mw)
                mixer = SideBySideSizes(left=_attention(_get(m, "left", dict, mw), mw + "left."),
                                        right=BonusSizes(_pos(right, "heads", mw + "right."), _pos(right, "dim", mw + "right.")))
            else:
                raise ConfigError(f"config.json {where}type {kind!r} is not a mixer of this design (known: 'mlstm', 'parallel')")
            layers.append(KavotarLayer(kind, mixer, _mlp(ly.get("mlp"), where + "mlp.")))
        cap = _get(d, "logit_softcap", float, "", required=False)
        return KavotarConfig(vocab=_pos(d, "vocab", ""), width=_pos(d, "width", ""), eps=_get(_get(d, "norm", dict, ""), "eps", float, "norm."),
                             logit_softcap=_positive(cap, "logit_softcap") if cap is not None else None, layers=tuple(layers))
