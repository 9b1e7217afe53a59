"""Kavotar as a model spec: blocks whose norms (layer norms) stand on the sublayers' results alone, around one of two mixers:
a matrix memory with exponential gates, or two mixers side by side, each normed over the width, half of their sum taken:
attention with a norm per head, a temperature per head, a partial rotation, a chunk mask and softmax weights mixed
across the heads, beside a decaying matrix state with token shift and a bonus for the current token.  Feed-forwards are
routed experts chosen by sigmoid scores with a correction, within the best groups.  The head has a matrix of its own, its
logits are capped.

Tensor names: ``embed``, ``head``, ``final.norm``; layer i under ``l<i>.``: ``norm1``, ``norm2``; memory ``mix.{q,k,v,g,o,norm,
i,i.b,f,f.b}``; side by side ``mix.left.{q,k,v,o,q.norm,k.norm,talk,temp,out}``, ``mix.right.{mu.r,mu.k,mu.v,mu.g,mu.w,r,k,v,g,
w1,w2,w0,u,norm,o,out}``; experts ``mlp.router``, ``mlp.correction``, ``mlp.e<j>.{gate,up,down}``.
"""
from __future__ import annotations

from ..config.kavotar_config import KavotarConfig, MemorySizes, SideBySideSizes
from ..config.registry import register_architecture
from ..parts.model import LayerSpec, ModelSpec

_ATTENTION_NAMES = {"q": ".q", "k": ".k", "v": ".v", "o": ".o", "q_norm": ".q.norm", "k_norm": ".k.norm", "temp": ".temp", "talk": ".talk"}


def _mixer(cfg: KavotarConfig, m):
    if isinstance(m, MemorySizes):
        return {"kind": "matrix_memory", "hidden": cfg.width, "heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap,
                "eps": cfg.eps}
    assert isinstance(m, SideBySideSizes)
    a, r = m.left, m.right
    position = ({"kind": "rope", "head_dim": a.dim, "rotary_dim": a.rot_dims, "theta": a.rot_base, "exact_frequencies": True}
                if a.rot_dims else {"kind": "none", "head_dim": a.dim})
    left = {"kind": "attention", "hidden": cfg.width, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim,
            "v_head_dim": a.vdim, "scale": a.scale, "window": None, "chunk": a.chunk, "head_norm": {"eps": cfg.eps, "weight": True},
            "head_scale": True, "talk": True, "position": position, "names": _ATTENTION_NAMES}
    right = {"kind": "token_mixing", "hidden": cfg.width, "heads": r.heads, "dim": r.dim, "eps": cfg.eps,
             "rank": None}  # the decay map's width is the checkpoint's
    return {"kind": "side_by_side", "left": left, "right": right, "left_scale": 0.5, "right_scale": 0.5,
            "out_norm": {"width": cfg.width, "eps": cfg.eps}}


def kavotar_spec(cfg: KavotarConfig) -> ModelSpec:
    norm = {"kind": "layernorm", "size": cfg.width, "eps": cfg.eps, "tensor_suffix": ""}
    layers, ignored = [], []
    for i, ly in enumerate(cfg.layers):
        f = ly.mlp
        ff = ({"kind": "routed_experts", "hidden": cfg.width, "experts": f.experts, "top": f.top, "intermediate": f.ff,
               "weights": "sigmoid", "groups": {"count": f.groups[0], "keep": f.groups[1]} if f.groups else None} if f else None)
        layers.append(LayerSpec(f"l{i}", {"kind": "result_norm", "norm": norm, "mixer": _mixer(cfg, ly.mixer), "feed_forward": ff}))
        if f is None:  # a layer without a feed-forward has no use for its second norm
            ignored.append(f"l{i}.norm2")
    return ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab, layers=layers, final_norm=norm, final_norm_prefix="final.norm",
        embedding={"kind": "token", "vocab": cfg.vocab, "hidden": cfg.width, "tensor": "embed"},
        head={"kind": "linear", "vocab": cfg.vocab, "hidden": cfg.width, "tensor": "head", "softcap": cfg.logit_softcap or 0.0},
        ignored_tensors=tuple(ignored),
    )


register_architecture("Kavotar", KavotarConfig.from_dict, kavotar_spec, model_type="kavotar")
