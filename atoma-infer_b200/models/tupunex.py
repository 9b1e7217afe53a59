"""Tupunex as a model spec: blocks on several residual streams side by side (hyper-connections, with a factor per channel on
every sublayer's result) around one of two mixers: differential attention without positions, inside a sliding window, with
biases, a short convolution on q, k and v, capped scores and a gate per head; or latent attention with a rotated key part
shared by all heads and a gate per head.  Feed-forwards are gated by SiLU.  The embedding is scaled; the head is a matrix of
its own.  A stretch of layers may run several times in a row with the same weights: every pass is a run of the schedule with a
cache and a state of its own.

Tensor names: ``embed``, ``final.norm``, ``head``; layer i under ``l<i>.``: ``norm1``, ``norm2``, ``ls1``, ``ls2``, ``hc1.in``, ``hc1.out``,
``hc1.mix`` and ``hc2.*``; differential attention ``mix.{q,k,v}`` with ``.b`` and ``.conv``, ``mix.{lq1,lk1,lq2,lk2,g,o}``; latent attention
``mix.{q,dkv,dkv.norm,uk,uv,g,o}``; feed-forward ``mlp.{gate,up,down}``.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.tupunex_config import DifferentialAttentionSizes, SharedLatentSizes, TupunexConfig
from ..parts.model import LayerRun, LayerSpec, ModelSpec

_NAMES = {"q": ".q", "k": ".k", "v": ".v", "o": ".o", "q_bias": ".q.b", "k_bias": ".k.b", "v_bias": ".v.b", "gate": ".g", "conv": ".conv"}


def _mixer(cfg: TupunexConfig, m):
    if isinstance(m, DifferentialAttentionSizes):
        return {"kind": "attention", "hidden": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                "v_head_dim": m.vdim, "scale": m.scale, "window": m.window, "softcap": m.softcap, "conv": m.conv, "bias": True,
                "head_gate": True, "differential": {"diff": m.diff, "eps": cfg.eps}, "names": _NAMES, "position": {"kind": "none"}}
    assert isinstance(m, SharedLatentSizes)
    return {"kind": "latent_attention", "hidden": cfg.width, "heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim,
            "v_head_dim": m.vdim, "q_rank": None, "kv_rank": m.kv_rank, "scale": m.scale, "window": None,
            "rotary_dims": m.rot_dims, "theta": m.rot_base, "halves": True, "eps": cfg.eps, "gate": "head"}


def tupunex_spec(cfg: TupunexConfig) -> ModelSpec:
    norm = {"kind": "rmsnorm", "size": cfg.width, "eps": cfg.eps, "tensor_suffix": ""}
    layers, ignored = [], []
    for i, ly in enumerate(cfg.layers):
        ff = ({"kind": "swiglu", "hidden": cfg.width, "intermediate": ly.mlp.ff, "names": {"gate": ".gate", "up": ".up", "down": ".down"}}
              if ly.mlp is not None else None)
        layers.append(LayerSpec(f"l{i}", {"kind": "hyper", "norm": norm, "mixer": _mixer(cfg, ly.mixer), "feed_forward": ff,
                                          "streams": cfg.streams}))
        if ly.mlp is None:  # a layer without a feed-forward has no use for what surrounds one
            ignored += [f"l{i}.{x}" for x in ("norm2", "ls2", "hc2.in", "hc2.out", "hc2.mix")]
    n, loop = len(layers), cfg.loop
    schedule = None
    if loop is not None:
        again = list(range(loop.start, loop.stop)) * loop.times
        schedule = [LayerRun(i) for i in list(range(loop.start)) + again + list(range(loop.stop, n))]
    return ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab, layers=layers, final_norm=norm, final_norm_prefix="final.norm",
        embedding={"kind": "token", "vocab": cfg.vocab, "hidden": cfg.width, "tensor": "embed", "scale": cfg.embedding_scale,
                   "copies": cfg.streams},
        head={"kind": "linear", "vocab": cfg.vocab, "hidden": cfg.width, "tensor": "head"},
        schedule=schedule, streams=cfg.streams, ignored_tensors=tuple(ignored),
    )


register_architecture("Tupunex", TupunexConfig.from_dict, tupunex_spec, model_type="tupunex")
