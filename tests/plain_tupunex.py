"""Tupunex, plainly: one function per mechanism, float64, whole sequences at once, written from the design's equations.

Shares no code with the engine.  ``forward(cfg, w, tokens)`` runs one request's tokens and returns the logits at every
position (and, on request, the sum of the streams after every layer run).  ``cfg`` is the configuration as config.json has
it (a dict), ``w`` a dict of tensors by checkpoint name.

Notation.  N(u) = u / sqrt(mean(u^2) + eps).  The model carries s streams X [T, s, width], all equal to the scaled
embedding at first.  A sublayer f with its weights a [s], M [s, s], b [s], its norm's weight n and its scale l:
Y = l * f(N(sum_j a_j X_j) * n);  X'_t = sum_j M[j, t] X_j + b_t Y.
"""
from __future__ import annotations

import torch

F = torch.float64

_ROUND = None   # a storage type that matrix products read and write through (None: exact), see ``forward``
_DITHER = None  # a generator that moves every value by up to half a unit of that type before it is rounded


def t64(x):
    return x.to(F)


def _rounded(x):
    if _DITHER is not None:
        x = x * (1.0 + torch.finfo(_ROUND).eps * (torch.rand(x.shape, generator=_DITHER, dtype=F) - 0.5))
    return x.to(_ROUND).to(F)


def stored(x):
    """A value that is kept in the storage type (exact if none is set)."""
    return x if _ROUND is None else _rounded(x)


def lin(x, w):
    """x W^T; with a storage type set, what the product reads and what it writes is rounded to that type."""
    return stored(stored(x) @ t64(w).T)


def unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit(x, eps) * t64(w)


def silu(z):
    return z * torch.sigmoid(z)


# ---------------------------------------------------------------------------------------------- streams
def read_streams(X, a):
    """X [T, s, width], a [s]: the weighted sum of the streams."""
    return torch.einsum("tsw,s->tw", X, t64(a))


def mix_streams(X, M, b, y):
    """M is indexed [from, to]; b says how much of the sublayer's result each stream takes."""
    return torch.einsum("tfw,fg->tgw", X, t64(M)) + t64(b)[None, :, None] * y[:, None, :]


# ---------------------------------------------------------------------------------------------- attention
def causal_conv(u, w):
    """u [T, C], w [C, taps]: out_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, C = u.shape
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=u.dtype), u], 0)
    out = torch.zeros_like(u)
    for j in range(taps):
        out = out + t64(w)[:, j] * padded[j:j + T]
    return out


def visible(T, window=None):
    """[T, T] bool: position i sees j <= i, with a window only those with i - j < window."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok if window is None else ok & (i - j < window)


def soft_limit(x, cap):
    return cap * torch.tanh(x / cap)


def softmax_over(scores, mask):
    """scores [..., T, T]; a row's weights over the keys its mask lets it see."""
    return torch.softmax(scores.masked_fill(~mask, float("-inf")), -1)


def two_maps(q, k, v, scale, cap, mask):
    """q [T, H, 2, d], k [T, G, 2, d], v [T, G, dv] -> [T, H, 2, dv]: per head two attentions over the same values."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        for m in range(2):
            s = (q[:, h, m] @ k[:, g, m].T) * scale
            if cap:
                s = soft_limit(s, cap)
            out.append(softmax_over(s, mask) @ v[:, g])
    return torch.stack(out, 1).reshape(q.shape[0], H, 2, v.shape[-1])


def map_weight(w, pre, diff):
    """What the second map is weighed with when it is taken off the first."""
    e = lambda a, b: torch.exp((t64(w[pre + a]) * t64(w[pre + b])).sum())  # noqa: E731
    return e("lq1", "lk1") - e("lq2", "lk2") + diff


def difference(a, lam, diff, eps):
    """a [T, H, 2, dv] -> [T, H, dv]."""
    return unit(a[:, :, 0] - lam * a[:, :, 1], eps) * (1.0 - diff)


def gate_heads(o, h, w_gate):
    """o [T, H, dv]: every head times one number of its own."""
    return o * torch.sigmoid(lin(h, w_gate))[:, :, None]


def differential_attention(m, w, pre, h, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rows = {}
    for x in "qkv":
        u = stored(lin(h, w[pre + x]) + t64(w[pre + x + ".b"]))
        rows[x] = stored(causal_conv(u, w[pre + x + ".conv"])) if m.get("conv") else u
    q, k, v = rows["q"].reshape(T, H, 2, d), rows["k"].reshape(T, G, 2, d), rows["v"].reshape(T, G, dv)
    a = stored(two_maps(q, k, v, m["scale"], m.get("softcap"), visible(T, (m.get("mask") or {}).get("size"))))
    o = difference(a, map_weight(w, pre, m["diff"]), m["diff"], eps)
    return lin(gate_heads(o, h, w[pre + "g"]).reshape(T, H * dv), w[pre + "o"])


# ---------------------------------------------------------------------------------------------- latent attention
def rotate_halves(x, dims, base):
    """x [T, ..., d]: dimension i pairs with i + dims / 2 (i < dims / 2) and turns by position * base^(-2i / dims)."""
    half = dims // 2
    ang = torch.arange(x.shape[0], dtype=F)[:, None] * base ** (-2.0 * torch.arange(half, dtype=F) / dims)[None, :]
    while ang.dim() < x.dim():
        ang = ang.unsqueeze(1)
    c, s = torch.cos(ang), torch.sin(ang)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def latent_attention(m, w, pre, h, eps):
    T, H, d, r, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m["rot"]
    q = lin(h, w[pre + "q"]).reshape(T, H, d + r)
    kv = lin(h, w[pre + "dkv"])
    c = stored(rms_norm(kv[:, :rank], w[pre + "dkv.norm"], eps))
    key_rot = stored(rotate_halves(kv[:, rank:], rot["dims"], rot["base"]))
    q_rot = stored(rotate_halves(q[:, :, d:], rot["dims"], rot["base"]))
    k = lin(c, w[pre + "uk"]).reshape(T, H, d)
    v = lin(c, w[pre + "uv"]).reshape(T, H, dv)
    see = visible(T)
    out = []
    for a in range(H):
        s = (q[:, a, :d] @ k[:, a].T + q_rot[:, a] @ key_rot.T) * m["scale"]
        out.append(softmax_over(s, see) @ v[:, a])
    o = stored(torch.stack(out, 1))
    return lin(gate_heads(o, h, w[pre + "g"]).reshape(T, H * dv), w[pre + "o"])


# ---------------------------------------------------------------------------------------------- the rest
def feed_forward(w, pre, h):
    return lin(silu(lin(h, w[pre + "gate"])) * lin(h, w[pre + "up"]), w[pre + "down"])


def layer_runs(cfg):
    """The layers in the order they run: a stretch of them may run several times in a row."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    inner = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + inner * loop["times"] + list(range(loop["stop"], n))


def forward(cfg, w, tokens, layers_out=None, round_to=None, dither=None):
    """``layers_out``: a list that receives the sum of the streams after every layer run; ``round_to``: a storage type
    through which every matrix product reads and writes (to see how far rounding alone moves a position); ``dither``: a
    seed; every value is moved by up to half a unit of that type first, another draw of the same roundings."""
    global _ROUND, _DITHER
    _ROUND, _DITHER = round_to, torch.Generator().manual_seed(dither) if dither is not None else None
    try:
        return _forward(cfg, w, tokens, layers_out)
    finally:
        _ROUND = _DITHER = None


def _forward(cfg, w, tokens, layers_out):
    eps = cfg["norm"]["eps"]
    x = t64(w["embed"])[torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    X = x[:, None, :].repeat(1, cfg["streams"], 1)
    for i in layer_runs(cfg):
        ly, p = cfg["layers"][i], f"l{i}."
        mixer = {"attention": differential_attention, "latent_attention": latent_attention}[ly["type"]]
        subs = [lambda h: mixer(ly["mixer"], w, p + "mix.", h, eps)]
        if ly.get("mlp") is not None:
            subs.append(lambda h: feed_forward(w, p + "mlp.", h))
        for q, f in enumerate(subs, 1):
            u = read_streams(X, w[p + f"hc{q}.in"])
            y = t64(w[p + f"ls{q}"]) * f(rms_norm(u, w[p + f"norm{q}"], eps))
            X = mix_streams(X, w[p + f"hc{q}.mix"], w[p + f"hc{q}.out"], y)
        if layers_out is not None:
            layers_out.append(X.sum(1))
    return lin(rms_norm(X.sum(1), w["final.norm"], eps), w["head"])
