"""Small Tupunex configurations for the tests, their model folders, and the plain logits of token lists.

The configurations differ in every size and constant and pick values that tell mechanisms apart: one stream, two, three, and
more than the kernels are built for by name; windows that are no multiple of a page, one that is shorter than a page, one
that is a multiple of it, and none; convolutions of one to five taps and none; maps narrower and wider than half of the
values, sizes that are no multiple of four; one key/value head for all heads and one for each; scores with a low cap, a
high one and none; rotations over part of the rotated part, all of it and none; a latent wider and narrower than what
it stands for; layers without a feed-forward; either kind of layer first; a stretch of layers that runs twice or three times,
from the first layer on, in the middle, up to the last layer, and no repetition at all.
"""
from __future__ import annotations

from typing import Dict, List

import torch

import helpers
import plain_tupunex as PX


def diff(heads, kv_heads, dim, vdim, scale, c, window=None, conv=None, softcap=None, ff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": c}
    if window:
        m["mask"] = {"size": window}
    if conv is not None:
        m["conv"] = conv
    if softcap:
        m["softcap"] = softcap
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, rot_dims=None, base=1e4, ff=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"dims": rot_dim if rot_dims is None else rot_dims, "base": base}}
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, streams, layers, loop=None, eps=1e-5, scale=1.0):
    c = {"architecture": "Tupunex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
         "streams": streams, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# name -> (config, page size)
CONFIGS = {
    # differential attention first: a window of 9 over pages of 4, four taps, values of twice a map, a low cap; the whole model
    # but its last layer runs twice; three streams; no feed-forward last
    "U": (config(96, 131, 3, [diff(4, 2, 16, 32, 0.5, 0.35, window=9, conv=4, softcap=3.0, ff=160),
                              latent(3, 16, 8, 24, 40, 0.4, ff=72),
                              diff(2, 1, 24, 16, 0.4, 0.8, window=30, conv=2, softcap=15.0)], loop=(0, 2, 2), scale=3.0), 4),
    # latent attention first, keys and values narrower than the latent; two streams; windows of 64 (a multiple of the page) and
    # none; a key/value head per head, no cap; three and no taps; the middle runs three times; head sizes of the tcgen05 kernels
    "V": (config(128, 300, 2, [latent(8, 16, 16, 16, 112, 0.3, base=500.0, ff=96),
                               diff(4, 4, 32, 64, 0.35, 0.2, window=64, conv=3, softcap=20.0, ff=200),
                               diff(6, 2, 64, 128, 0.25, 0.5, conv=0, ff=64)], loop=(1, 2, 3), eps=1e-6, scale=0.5), 16),
    # sizes that are no multiple of four (maps of 9, values of 10, a latent of 21 beside 6, of which 4 turn); a window of 5 below
    # the page of 8, one tap; more streams than any kernel names; the loop ends with the last layer
    "W": (config(70, 97, 6, [diff(3, 1, 9, 10, 0.7, 0.6, window=5, conv=1, softcap=6.0, ff=50),
                             latent(2, 10, 6, 14, 21, 0.6, rot_dims=4, base=50.0),
                             diff(4, 2, 18, 30, 0.4, 0.3, window=21, conv=5, ff=44),
                             latent(5, 8, 2, 6, 30, 0.5, rot_dims=0, ff=30)], loop=(2, 4, 2), scale=2.0), 8),
    # one stream, no repetition, two latent layers in a row; ten heads over one key/value head (twenty query maps a key head:
    # more than a tile of the tensor-core kernels takes)
    "X": (config(64, 111, 1, [latent(4, 12, 12, 20, 24, 0.5, ff=40), latent(1, 24, 8, 32, 56, 0.35),
                              diff(10, 1, 8, 16, 0.6, 0.45, window=17, conv=3, softcap=8.0, ff=56)], scale=1.5), 8),
}

# stds that make every mechanism matter and leave the streams near 1: biases of order one, convolutions far from zero, maps
# whose weights differ, gates that open and close, queries that choose among keys.  A key counts wherever it is part of a
# name, and the factors of all keys that match multiply.
SCALES = {".q.b": 12.0, ".k.b": 12.0, ".v.b": 12.0, ".conv": 9.0, ".lq": 5.0, ".lk": 5.0, "mix.g": 4.0, "mix.q": 2.5, "mix.k": 2.5, "mix.dkv": 2.0,
          "mix.u": 2.0, "embed": 12.0, "head": 2.0}


def make_model(path: str, name: str, seed: int = 0) -> str:
    """Streams are read and mixed with weights well apart from the sum and the identity; what a sublayer's result is
    multiplied by lies between 0.3 and 0.9."""
    import os

    from atoma_infer_b200.weights.safetensors_io import write_safetensors

    cfg, _ = CONFIGS[name]
    d = helpers.make_model(path, cfg, seed=seed, scales=SCALES, norm_jitter=0.25)
    w = helpers.read_weights(d)
    for k in w:
        if ".ls" in k:
            w[k] = 0.3 + 0.6 * torch.sigmoid(4.0 * (w[k] - 1.0))
        if ".mix" in k and ".hc" in k:  # rows that keep a stream's size, with much of each stream handed to the others
            s = w[k].shape[0]
            w[k] = 0.75 * w[k] + 0.25 / s
    write_safetensors(os.path.join(d, "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in w.items()}, {})
    return d


def plain_logits(model_dir: str, cfg: dict, seqs: Dict[str, List[int]]) -> Dict[str, torch.Tensor]:
    w = helpers.read_weights(model_dir)
    return {k: PX.forward(cfg, w, v) for k, v in seqs.items()}


def plain_greedy(model_dir: str, cfg: dict, prompt: List[int], n: int) -> List[int]:
    w = helpers.read_weights(model_dir)
    toks, out = list(prompt), []
    for _ in range(n):
        t = int(torch.argmax(PX.forward(cfg, w, toks)[-1]))
        out.append(t)
        toks.append(t)
    return out


def rounding_errors(model_dir: str, cfg: dict, seqs: Dict[str, List[int]], ref: Dict[str, torch.Tensor],
                    dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Per position, how far the plain implementation itself moves (largest logit difference over the largest logit of
    the sequence, the largest of three draws of the roundings) when what its matrix products read and write is rounded to
    ``dtype``: the measure of how much a position amplifies roundings that no implementation in that type can avoid.
    (float32: twice that, since a product's sum is then rounded at every step and not once.)"""
    w = helpers.read_weights(model_dir)
    f = 2.0 if dtype == torch.float32 else 1.0
    worst = lambda k, v: torch.stack([(PX.forward(cfg, w, v, round_to=dtype, dither=s) - ref[k]).abs().max(-1).values  # noqa: E731
                                      for s in (None, 1, 2)]).max(0).values
    return {k: f * worst(k, v) / ref[k].abs().max() for k, v in seqs.items()}
