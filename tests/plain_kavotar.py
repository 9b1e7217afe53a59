"""Kavotar, plainly: one function per mechanism, float64, whole sequences at once, written from the design's equations.

Shares no code with the engine.  ``forward(cfg, w, tokens)`` runs one request's tokens and returns the logits at every
position (and, on request, the stream after every layer).  ``cfg`` is the configuration as config.json has it (a
dict), ``w`` a dict of tensors by checkpoint name.

Notation.  L(u) = (u - mean u) / sqrt(mean((u - mean u)^2) + eps) * w, N(u) = u / sqrt(mean(u^2) + eps).  A layer:
x <- x + L1(mixer(x)); x <- x + L2(experts(x)).
"""
from __future__ import annotations

import math

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


def lin(x, w):
    """x W^T; with a storage type set, what the product reads and what it writes is rounded to that type first."""
    if _ROUND is None:
        return x @ t64(w).T
    return _rounded(_rounded(x) @ t64(w).T)


def lin_wide(x, w):
    """Like ``lin``, with a result that is not rounded (what enters a recurrence's gates, a router)."""
    return (x if _ROUND is None else _rounded(x)) @ t64(w).T


def layer_norm(x, w, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * t64(w)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


# ---------------------------------------------------------------------------------------------- attention
def rotate_halves(x, dims, base):
    """x [T, heads, dim]: dimension i pairs with i + dims / 2 (i < dims / 2) and turns by p * base^(-2i / dims)."""
    if not dims:
        return x
    half = dims // 2
    i = torch.arange(half, dtype=F)
    ang = torch.arange(x.shape[0], dtype=F)[:, None] * base ** (-2.0 * i / dims)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    out = x.clone()
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def visible(T, chunk=None):
    """[T, T] bool: position i sees j <= i, with chunks only those of its own."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok if chunk is None else ok & (torch.div(i, chunk, rounding_mode="floor") == torch.div(j, chunk, rounding_mode="floor"))


def head_weights(q, k, scale, temp, mask):
    """q [T, H, d], k [T, G, d] -> softmax weights [H, T, T] of (q . k) * scale * temp_h over the visible keys."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros((H, T, T), dtype=F)
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // G)].T) * scale * temp[h]
        out[h] = torch.softmax(s.masked_fill(~mask, -math.inf), -1)
    return out


def mix_heads(weights, talk):
    """weights [H, T, T]: head h's become sum_g talk[h, g] weights_g."""
    return torch.einsum("hg,gij->hij", t64(talk), weights)


def weighted_values(weights, v):
    """weights [H, T, T], v [T, G, dv] -> [T, H, dv]: head h weighs the values of key/value head h // (H / G)."""
    H, G = weights.shape[0], v.shape[1]
    return torch.stack([weights[h] @ v[:, h // (H // G)] for h in range(H)], 1)


def attention(m, w, pre, x, eps):
    T = x.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(lin(x, w[pre + "q"]).view(T, H, d), eps) * t64(w[pre + "q.norm"])
    k = rms(lin(x, w[pre + "k"]).view(T, G, d), eps) * t64(w[pre + "k.norm"])
    v = lin(x, w[pre + "v"]).view(T, G, dv)
    rot = m.get("rot")
    if rot:
        q, k = rotate_halves(q, rot["dims"], rot["base"]), rotate_halves(k, rot["dims"], rot["base"])
    if _ROUND is not None:
        q, k = _rounded(q), _rounded(k)
    mask = m.get("mask")
    p = head_weights(q, k, m["scale"], t64(w[pre + "temp"]), visible(T, mask["size"] if mask else None))
    o = weighted_values(mix_heads(p, w[pre + "talk"]), v)
    return lin(o.reshape(T, H * dv), w[pre + "o"])


# ---------------------------------------------------------------------------------------------- token mixing with a decaying matrix
def moved_toward_previous(x, mu):
    before = torch.cat([torch.zeros_like(x[:1]), x[:-1]], 0)
    return x + (before - x) * t64(mu)


def bonus_state(r, k, v, decay, u):
    """Per head o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t, then S_t = diag(decay_t) S_(t-1) + k_t v_t^T; r, k, decay
    [T, H, d], v [T, H, dv], u [H, d]."""
    T, H, d = r.shape
    out = torch.zeros((T, H, v.shape[2]), dtype=F)
    for h in range(H):
        S = torch.zeros((d, v.shape[2]), dtype=F)
        for t in range(T):
            kv = k[t, h][:, None] * v[t, h][None, :]
            out[t, h] = (S + u[h][:, None] * kv).T @ r[t, h]
            S = decay[t, h][:, None] * S + kv
    return out


def token_mixing(m, w, pre, x, eps):
    T = x.shape[0]
    H, d = m["heads"], m["dim"]
    mix = {s: moved_toward_previous(x, w[pre + "mu." + s]) for s in "rkvgw"}
    r, k, v = (lin(mix[s], w[pre + s]).view(T, H, d) for s in "rkv")
    gate = silu(lin(mix["g"], w[pre + "g"]))
    z = lin_wide(torch.tanh(lin(mix["w"], w[pre + "w1"])), w[pre + "w2"]) + t64(w[pre + "w0"])
    decay = torch.exp(-torch.exp(z)).view(T, H, d)
    o = rms(bonus_state(r, k, v, decay, t64(w[pre + "u"])), eps).reshape(T, H * d)
    return lin(o * t64(w[pre + "norm"]) * gate, w[pre + "o"])


def parallel(m, w, pre, x, eps):
    left = rms(attention(m["left"], w, pre + "left.", x, eps), eps) * t64(w[pre + "left.out"])
    right = rms(token_mixing(m["right"], w, pre + "right.", x, eps), eps) * t64(w[pre + "right.out"])
    return 0.5 * (left + right)


# ---------------------------------------------------------------------------------------------- matrix memory with exponential gates
def matrix_memory(q, k, v, log_i, log_f):
    """Per head, with the running maximum m (0 at the start): m' = max(f + m, i); S <- exp(f + m - m') S + exp(i - m') k v^T,
    n likewise with k alone; o = S^T q / (max(|n . q|, exp(-m')) + 1e-6).  q, k [T, H, d], v [T, H, dv], gates [T, H]."""
    T, H, d = q.shape
    out = torch.zeros((T, H, v.shape[2]), dtype=F)
    for h in range(H):
        S, n, m = torch.zeros((d, v.shape[2]), dtype=F), torch.zeros(d, dtype=F), torch.zeros((), dtype=F)
        for t in range(T):
            i, f = log_i[t, h], log_f[t, h]
            new = torch.maximum(f + m, i)
            keep, take = torch.exp(f + m - new), torch.exp(i - new)
            S = keep * S + take * k[t, h][:, None] * v[t, h][None, :]
            n = keep * n + take * k[t, h]
            m = new
            out[t, h] = (S.T @ q[t, h]) / (torch.maximum((n @ q[t, h]).abs(), torch.exp(-m)) + 1e-6)
    return out


def soft_limit(z, cap):
    return cap * torch.tanh(z / cap)


def log_sigmoid(z):
    return -torch.nn.functional.softplus(-z)


def mlstm(m, w, pre, x, eps):
    T = x.shape[0]
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = lin(x, w[pre + "q"]).view(T, H, d) * d ** -0.5
    k = lin(x, w[pre + "k"]).view(T, H, d)
    v = lin(x, w[pre + "v"]).view(T, H, dv)
    log_i = soft_limit(lin_wide(x, w[pre + "i"]) + t64(w[pre + "i.b"]), cap)
    log_f = log_sigmoid(soft_limit(lin_wide(x, w[pre + "f"]) + t64(w[pre + "f.b"]), cap))
    o = rms(matrix_memory(q, k, v, log_i, log_f), eps).reshape(T, H * dv)
    return lin(o * t64(w[pre + "norm"]) * torch.sigmoid(lin(x, w[pre + "g"])), w[pre + "o"])


# ---------------------------------------------------------------------------------------------- experts
def choose(s, correction, top, groups=None, margins=None):
    """s [T, E] sigmoid scores -> (experts [T, top], weights [T, top]).  Choice by s + correction; with ``groups``
    ({"count", "keep"}) only experts of the ``keep`` groups whose two largest choice scores sum highest."""
    c = s + t64(correction)
    T, E = c.shape
    lead = torch.full((T,), math.inf, dtype=F)
    if groups:
        n, keep = groups["count"], groups["keep"]
        per = E // n
        g = torch.topk(c.view(T, n, per), min(2, per), dim=-1).values.sum(-1)
        order = torch.sort(g, dim=-1, descending=True, stable=True)
        if keep < n:
            lead = torch.minimum(lead, order.values[:, keep - 1] - order.values[:, keep])
        kept = torch.zeros((T, n), dtype=torch.bool).scatter(1, order.indices[:, :keep], True)
        c = c.masked_fill(~kept.repeat_interleave(per, 1), -math.inf)
    order = torch.sort(c, dim=-1, descending=True, stable=True)
    if top < E:
        lead = torch.minimum(lead, order.values[:, top - 1] - order.values[:, top])
    if margins is not None:
        margins.append(lead)
    idx = order.indices[:, :top]
    return idx, torch.gather(s, 1, idx)


def experts(f, w, pre, x, margins=None):
    r = f["router"]
    s = torch.sigmoid(lin_wide(x, w[pre + "router"]))
    idx, wt = choose(s, w[pre + "correction"], r["top"], r.get("groups"), margins)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for c in range(idx.shape[1]):
            e = pre + f"e{int(idx[t, c])}."
            y = silu(lin(x[t], w[e + "gate"])) * lin(x[t], w[e + "up"])
            out[t] = out[t] + wt[t, c] * lin(y, w[e + "down"])
    return out


# ---------------------------------------------------------------------------------------------- the model
def forward(cfg, w, tokens, layers_out=None, margins=None, round_to=None, dither=None):
    """``layers_out``: a list that receives the stream after every layer; ``margins``: a list that receives, per routed
    layer, by how much every position's choice of experts (and of groups) leads what was not chosen; ``round_to``: a
    storage type through which every matrix product reads and writes (to see how far rounding alone moves a position);
    ``dither``: a seed; every value is moved by up to half a unit of that type first, another draw of the same roundings."""
    global _ROUND, _DITHER
    _ROUND, _DITHER = round_to, torch.Generator().manual_seed(dither) if dither is not None else None
    try:
        return _forward(cfg, w, tokens, layers_out, margins)
    finally:
        _ROUND = _DITHER = None


def _forward(cfg, w, tokens, layers_out, margins):
    eps = cfg["norm"]["eps"]
    x = t64(w["embed"])[torch.as_tensor(tokens, dtype=torch.long)]
    for i, ly in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = {"mlstm": mlstm, "parallel": parallel}[ly["type"]]
        x = x + layer_norm(mixer(ly["mixer"], w, p + "mix.", x, eps), w[p + "norm1"], eps)
        if ly.get("mlp") is not None:
            x = x + layer_norm(experts(ly["mlp"], w, p + "mlp.", x, margins), w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    z = lin(layer_norm(x, w["final.norm"], eps), w["head"])
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z
