"""Small Kavotar configurations for the tests, their model folders, and the plain logits of token lists.

The configurations differ in every size and constant and pick values that tell mechanisms apart: chunks that are a
multiple of a page, that are none, that are shorter than a page, and none at all; a rotation over part of a head, over
all of it and none, with sizes that are no multiple of four; heads of keys larger and smaller than heads of values; one
key/value head for all query heads and one for each; one recurrent head and several; memories wider than tall and
taller than wide, with gates capped low and high; experts in groups of one, two and more of which some or all are kept, and
in no groups; one, some or all experts chosen; a layer without a feed-forward; either kind of layer first; logits with and
without cap.
"""
from __future__ import annotations

from typing import Dict, List

import torch

import helpers
import plain_kavotar as PV
from kulivik_helpers import want_before  # noqa: F401  (the same for every routed design)


def memory(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def talking(heads, kv_heads, dim, vdim, scale, chunk=None, rot=None, base=1e4):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk:
        m["mask"] = {"size": chunk}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
    return m


def pair(left, heads, dim):
    return {"left": left, "right": {"heads": heads, "dim": dim}}


def moe(ff, experts, top, groups=None):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(width, vocab, layers, eps=1e-5, logit_softcap=None):
    c = {"architecture": "Kavotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if logit_softcap is not None:
        c["logit_softcap"] = logit_softcap
    return c


# name -> (config, page size)
CONFIGS = {
    # the memory first, wider than tall; chunks of 12 over pages of 4, half a head rotated; groups of two; no feed-forward last
    "U": (config(96, 131, [layer("mlstm", memory(3, 16, 40, 6.0), moe(40, 8, 2, (4, 2))),
                           layer("parallel", pair(talking(6, 3, 32, 16, 0.3, chunk=12, rot=16, base=200.0), 3, 24), moe(48, 6, 3, (3, 2))),
                           layer("mlstm", memory(1, 48, 24, 2.5))], logit_softcap=12.0), 4),
    # side by side first: one key/value head for eight query heads, no chunks, the whole head rotated; all experts chosen;
    # then a key/value head per query head, chunks shorter than a page, no rotation; groups of one; logits as they are
    "V": (config(128, 300, [layer("parallel", pair(talking(8, 1, 16, 48, 0.4, rot=16, base=1e6), 2, 40), moe(24, 3, 3)),
                            layer("mlstm", memory(4, 32, 16, 20.0), moe(64, 6, 2, (6, 3))),
                            layer("parallel", pair(talking(4, 4, 64, 64, 0.2, chunk=10), 1, 72), moe(32, 4, 1, (2, 1)))], eps=1e-6), 16),
    # sizes that are no multiple of four (heads of 18 with 6 rotated, values of 10, memories of 10 x 14); chunks of 25 that
    # no page divides; three layers of the side-by-side kind, two in a row
    "W": (config(72, 97, [layer("parallel", pair(talking(4, 2, 18, 10, 0.35, chunk=25, rot=6, base=50.0), 2, 12), moe(32, 9, 4, (3, 3))),
                          layer("mlstm", memory(2, 10, 14, 9.0), moe(16, 12, 5, (4, 2))),
                          layer("parallel", pair(talking(5, 5, 16, 16, 0.25, chunk=64, rot=2), 3, 18), moe(20, 2, 1)),
                          layer("parallel", pair(talking(2, 1, 24, 32, 0.3, chunk=7, rot=24), 1, 8), moe(56, 5, 2, (5, 4)))],
                 logit_softcap=25.0), 8),
}

# stds that make every mechanism matter and leave the stream near 1: shifts well inside (0, 1), decays from fast to slow,
# gates that open and close, mixing across heads of order one, corrections that turn choices, routers that choose clearly.
# A key counts wherever it is part of a name, and the factors of all keys that match multiply.
SCALES = {".mu.": 10.0, ".w0": 25.0, "right.w1": 4.0, "right.w2": 6.0, ".u": 12.0, ".talk": 10.0, ".temp": 1.0, "correction": 2.0,
          "router": 6.0, ".i.b": 20.0, ".f.b": 30.0, "mix.i": 4.0, "mix.f": 4.0, "mix.q": 3.0, "mix.k": 3.0, "left.q": 2.0, "right.r": 3.0,
          "right.k": 3.0, "embed": 12.0, "head": 2.0}


def make_model(path: str, name: str, seed: int = 0, decisive: bool = False) -> str:
    """What reads a matrix state (q of a memory, r of a token mixing) is drawn near what was written to it (k), and the bonus
    is positive: a token finds itself, so no head's output is a near cancellation that its norm would blow up, whatever the
    number format.  ``decisive``: corrections so far apart that the same experts of every layer run for every token: no choice
    hangs on a lead that rounding to bfloat16 can turn (how choices follow the tokens is tested in float32)."""
    import os

    from atoma_infer_b200.weights.safetensors_io import write_safetensors

    cfg, _ = CONFIGS[name]
    d = helpers.make_model(path, cfg, seed=seed, scales=SCALES, norm_jitter=0.2)
    w = helpers.read_weights(d)
    for i, ly in enumerate(cfg["layers"]):
        read, written = (f"l{i}.mix.q", f"l{i}.mix.k") if ly["type"] == "mlstm" else (f"l{i}.mix.right.r", f"l{i}.mix.right.k")
        w[read] = w[written] + 0.4 * w[read]
        if ly["type"] == "parallel":  # (both read nearly the same row too)
            w[f"l{i}.mix.right.mu.r"] = w[f"l{i}.mix.right.mu.k"] + 0.3 * w[f"l{i}.mix.right.mu.r"]
            w[f"l{i}.mix.right.u"] = w[f"l{i}.mix.right.u"].abs() + 0.3
        if decisive and ly.get("mlp"):
            r = ly["mlp"]["router"]
            n = r.get("groups", {}).get("count", 1)
            order = torch.randperm(n, generator=torch.Generator().manual_seed(seed + i))
            per = r["experts"] // n
            inside = torch.stack([torch.randperm(per, generator=torch.Generator().manual_seed(100 * seed + 10 * i + g)) for g in range(n)])
            w[f"l{i}.mlp.correction"] = (1.25 * (order[:, None] * per + inside) - 4.0).reshape(-1)
    write_safetensors(os.path.join(d, "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in w.items()}, {})
    return d


def plain_logits(model_dir: str, cfg: dict, seqs: Dict[str, List[int]]) -> Dict[str, torch.Tensor]:
    w = helpers.read_weights(model_dir)
    return {k: PV.forward(cfg, w, v) for k, v in seqs.items()}


def plain_greedy(model_dir: str, cfg: dict, prompt: List[int], n: int) -> List[int]:
    w = helpers.read_weights(model_dir)
    toks, out = list(prompt), []
    for _ in range(n):
        t = int(torch.argmax(PV.forward(cfg, w, toks)[-1]))
        out.append(t)
        toks.append(t)
    return out


def first_close_call(model_dir: str, cfg: dict, seqs: Dict[str, List[int]], lead: float = 0.02) -> Dict[str, int]:
    """Per request the first position at which a router's choice (of experts or of groups) hangs on a lead of less than
    ``lead`` (the length of the request if there is none).  From there on a reduced-precision engine may rightly choose
    another expert, and every later position of the request reads what that choice left in the caches."""
    w = helpers.read_weights(model_dir)
    out = {}
    for k, v in seqs.items():
        margins: list = []
        PV.forward(cfg, w, v, margins=margins)
        worst = torch.stack(margins).min(0).values if margins else torch.full((len(v),), float("inf"))
        close = (worst < lead).nonzero().flatten()
        out[k] = int(close[0]) if len(close) else len(v)
    return out


def rounding_errors(model_dir: str, cfg: dict, seqs: Dict[str, List[int]], ref: Dict[str, torch.Tensor],
                    dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Per position, how far the plain implementation itself moves (largest logit difference over the largest logit of
    the sequence, the largest of three draws of the roundings) when what its matrix products read and write is rounded to
    ``dtype``: the measure of how much a position amplifies roundings that no implementation in that type can avoid.
    (float32: twice that, since a product's sum is then rounded at every step and not once.)"""
    w = helpers.read_weights(model_dir)
    f = 2.0 if dtype == torch.float32 else 1.0
    worst = lambda k, v: torch.stack([(PV.forward(cfg, w, v, round_to=dtype, dither=s) - ref[k]).abs().max(-1).values  # noqa: E731
                                      for s in (None, 1, 2)]).max(0).values
    return {k: f * worst(k, v) / ref[k].abs().max() for k, v in seqs.items()}
