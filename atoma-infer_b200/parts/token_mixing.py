"""Time mixing of the RWKV kind: a matrix of dim x dim per head that decays row by row, read before the current token enters
it, with a bonus for that token.

With x' the request's row before x (zeros before its first token) each of r, k, v, g, w reads a row of its own,
x + (x' - x) * mu_s.  r, k, v = W_r, W_k, W_v of their rows (heads x dim), gate = silu(W_g of its row); the decay of key
channel n of a head is exp(-exp(z)), z = W_w2 tanh(W_w1 of its row) + w0.  Per head o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t,
then S_t = diag(decay_t) S_(t-1) + k_t v_t^T.  Each head's o is divided by its root mean square; the heads side by side are
multiplied by a weight of their size and by the gate, and projected out.

State per request (float32, fixed size, ``cache.state[slot]``): the row before (the first share), then the heads' matrices
[heads, dim, dim], zero at the start; no pages.  The rows are the float32 ones where the block hands them over
(``ctx.shared["mixer_rows"]``).  The shift, the decay (its logits leave their projection as float32), the recurrence, the
norm and the gate are float32 in every mode; the projections run in the compute dtype.

Parameters: ``hidden``, ``heads``, ``dim``, ``rank`` (of the decay's map; None: whatever the checkpoint's tensors have, 16 in
random-weights mode), ``eps``, ``names`` (suffixes of the tensors: mu, r, k, v, g, w1, w2, w0, u, norm, o).
"""
from __future__ import annotations

import torch

from ..config.registry import register_part
from ..weights.loader import FreeDim, TensorDecl
from .base import Mixer

_NAMES = {"mu": ".mu.", "r": ".r", "k": ".k", "v": ".v", "g": ".g", "w1": ".w1", "w2": ".w2", "w0": ".w0", "u": ".u", "norm": ".norm", "o": ".o"}


class TokenMixing(Mixer):
    graph_safe = True  # reads the step's metadata on the device only

    def __init__(self, params, prefix):
        super().__init__(params, prefix)
        p = params
        self.hidden, self.heads, self.dim, self.eps = int(p["hidden"]), int(p["heads"]), int(p["dim"]), float(p["eps"])
        self.rank = int(p["rank"]) if p.get("rank") is not None else FreeDim(prefix + ":decay rank", 16)
        self.names = {**_NAMES, **(p.get("names") or {})}
        self.inner = self.heads * self.dim

    def _kept(self):
        """Floats of the kept row, rounded up so that the matrices start on 16 bytes."""
        return -(-self.hidden // 4) * 4

    def state_bytes(self):
        return (self._kept() + self.inner * self.dim) * 4

    def activation_width(self):
        return 5 * self.hidden + 4 * self.inner + 5 * self.inner

    def declare(self):
        pre, n, W, I = self.prefix, self.names, self.hidden, self.inner
        return ([TensorDecl(pre + n["mu"] + s, (W,)) for s in "rkvgw"] + [TensorDecl(pre + n[s], (I, W)) for s in "rkvg"]
                + [TensorDecl(pre + n["w1"], (self.rank, W)), TensorDecl(pre + n["w2"], (I, self.rank)), TensorDecl(pre + n["w0"], (I,)),
                   TensorDecl(pre + n["u"], (self.heads, self.dim)), TensorDecl(pre + n["norm"], (I,), init="ones"),
                   TensorDecl(pre + n["o"], (W, I))])

    def bind(self, tensors, rt):
        super().bind(tensors, rt)
        pre, n = self.prefix, self.names
        t = lambda name: tensors[pre + n[name]]  # noqa: E731
        f32 = lambda x: x.to(torch.float32).contiguous()  # noqa: E731  (exact widening)
        self.mu = f32(torch.stack([tensors[pre + n["mu"] + s] for s in "rkvgw"]))
        self.w_in = torch.stack([t(s) for s in "rkvg"]).contiguous()  # [4, inner, hidden], each reads a row of its own
        self.w1, self.w2, self.w_out = t("w1").contiguous(), t("w2").contiguous(), t("o").contiguous()
        self.w0, self.bonus, self.norm_w = f32(t("w0")), f32(t("u").reshape(-1)), f32(t("norm"))

    def streamed_weights(self):
        return [*self.w_in, self.w1, self.w2, self.w_out]

    def states(self, state):
        """The per-request state as float32 views: the kept rows [slots, hidden], the matrices [slots, heads, dim, dim]."""
        f = state[:, :self.state_bytes()].view(torch.float32)
        a = self._kept()
        return f[:, :self.hidden], f[:, a:a + self.inner * self.dim].view(f.shape[0], self.heads, self.dim, self.dim)

    def forward(self, x, ctx, cache):
        ops, T, W, I = self.rt.ops, ctx.T, self.hidden, self.inner
        kept, matrices = self.states(cache.state)
        rows = ctx.shared.get("mixer_rows")
        rows = x if rows is None else rows
        mixed = torch.empty((5, T, W), dtype=x.dtype, device=x.device)
        if not ops.token_mix(rows, self.mu, kept, ctx, mixed):
            ops.keep_last_rows(rows, kept, ctx)  # after the rows before have been read
        r, k, v, g = ops.linears(mixed[:4], self.w_in, meta=ctx.meta)
        low = ops.linear(mixed[4], self.w1, out_dtype=torch.float32, meta=ctx.meta)
        act = torch.empty(low.shape, dtype=x.dtype, device=x.device)
        ops.tanh_rows(low, act, ctx.meta)
        z = ops.linear(act, self.w2, out_dtype=torch.float32, meta=ctx.meta)
        o = torch.empty((T, I), dtype=torch.float32, device=x.device)
        ops.bonus_scan(r, k, v, z, self.w0, self.bonus, matrices, ctx, o, heads=self.heads, dim=self.dim, vdim=self.dim)
        y = torch.empty((T, I), dtype=x.dtype, device=x.device)
        ops.head_weight_norm_gate(o, g, self.norm_w, self.eps, y, ctx.meta, self.heads, kind="silu")
        return ops.linear(y, self.w_out, meta=ctx.meta)


register_part("mixer", "token_mixing", TokenMixing)
