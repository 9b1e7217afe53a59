"""Matrix memory with exponential gates (the mLSTM of xLSTM): a matrix and a normalizer per head.

q = W_q x * dim^(-1/2), k = W_k x (heads x dim), v = W_v x (heads x vdim).  Per head a log input gate i = cap tanh((W_i x +
b_i) / cap) and a log forget gate f = log sigmoid(cap tanh((W_f x + b_f) / cap)).  With a running maximum m (0 at the start):
m_t = max(f + m_(t-1), i); S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k_t v_t^T, n_t likewise with k_t alone;
o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6).  Each head's o is divided by its root mean square; the heads side by
side are multiplied by a weight of their size and by sigmoid(W_g x), and projected out.

State per request (float32, fixed size, ``cache.state[slot]``): the heads' matrices [heads, dim, vdim], normalizers [heads,
dim] and maxima [heads], zero at the start; no pages.  The gates (their logits leave the projection as float32), the
recurrence, the division, the norm and the output gate are float32 in every mode.

Parameters: ``hidden``, ``heads``, ``dim``, ``vdim``, ``gate_cap``, ``eps``, ``names`` (suffixes of the tensors: q, k, v, g, o,
norm, i, f, i_bias, f_bias).
"""
from __future__ import annotations

import torch

from ..config.registry import register_part
from ..weights.loader import TensorDecl
from .base import Mixer

_NAMES = {"q": ".q", "k": ".k", "v": ".v", "g": ".g", "o": ".o", "norm": ".norm", "i": ".i", "f": ".f", "i_bias": ".i.b", "f_bias": ".f.b"}


class MatrixMemory(Mixer):
    graph_safe = True  # reads the step's metadata on the device only

    def __init__(self, params, prefix):
        super().__init__(params, prefix)
        p = params
        self.hidden, self.heads, self.dim, self.vdim = int(p["hidden"]), int(p["heads"]), int(p["dim"]), int(p["vdim"])
        self.cap, self.eps = float(p["gate_cap"]), float(p["eps"])
        if self.cap <= 0:
            raise ValueError("gate_cap must be positive")
        self.names = {**_NAMES, **(p.get("names") or {})}
        self.qk, self.vg = self.heads * self.dim, self.heads * self.vdim

    def _shares(self):
        """Floats of the matrices (rounded up so that what follows starts on 16 bytes), of the normalizers, of the maxima."""
        up = lambda n: -(-n // 4) * 4  # noqa: E731
        return up(self.qk * self.vdim), up(self.qk), up(self.heads)

    def state_bytes(self):
        return sum(self._shares()) * 4

    def activation_width(self):
        return 2 * self.qk + 2 * self.vg + 2 * self.vg + 12 * self.heads

    def declare(self):
        pre, n = self.prefix, self.names
        return [
            TensorDecl(pre + n["q"], (self.qk, self.hidden)), TensorDecl(pre + n["k"], (self.qk, self.hidden)),
            TensorDecl(pre + n["v"], (self.vg, self.hidden)), TensorDecl(pre + n["g"], (self.vg, self.hidden)),
            TensorDecl(pre + n["o"], (self.hidden, self.vg)), TensorDecl(pre + n["norm"], (self.vg,), init="ones"),
            TensorDecl(pre + n["i"], (self.heads, self.hidden)), TensorDecl(pre + n["i_bias"], (self.heads,)),
            TensorDecl(pre + n["f"], (self.heads, self.hidden)), TensorDecl(pre + n["f_bias"], (self.heads,)),
        ]

    def bind(self, tensors, rt):
        super().bind(tensors, rt)
        pre, n = self.prefix, self.names
        t = lambda name: tensors[pre + n[name]]  # noqa: E731
        self.w_in = torch.cat([t("q"), t("k"), t("v"), t("g")], dim=0).contiguous()
        self.w_gates = torch.cat([t("i"), t("f")], dim=0).contiguous()  # apart: their logits stay float32
        self.b_gates = torch.cat([t("i_bias"), t("f_bias")]).to(torch.float32).contiguous()  # widened exactly
        self.w_out = t("o").contiguous()
        self.norm_w = t("norm").to(torch.float32).contiguous()

    def streamed_weights(self):
        return [self.w_in, self.w_gates, self.w_out]

    def states(self, state):
        """The per-request state as float32 views: matrices [slots, heads, dim, vdim], normalizers [slots, heads, dim],
        maxima [slots, heads]."""
        a, b, _ = self._shares()
        f = state[:, :self.state_bytes()].view(torch.float32)
        S = f.shape[0]
        return (f[:, :self.qk * self.vdim].view(S, self.heads, self.dim, self.vdim), f[:, a:a + self.qk].view(S, self.heads, self.dim),
                f[:, a + b:a + b + self.heads])

    def forward(self, x, ctx, cache):
        ops, T, qk, vg = self.rt.ops, ctx.T, self.qk, self.vg
        proj = ops.linear(x, self.w_in, meta=ctx.meta)
        logits = ops.linear(x, self.w_gates, out_dtype=torch.float32, meta=ctx.meta)
        f32 = lambda *shape: torch.empty(shape, dtype=torch.float32, device=x.device)  # noqa: E731
        o, nq, floor = f32(T, vg), f32(T, self.heads), f32(T, self.heads)
        ops.memory_scan(proj[:, :qk], proj[:, qk:2 * qk], proj[:, 2 * qk:2 * qk + vg], logits, self.b_gates, self.cap,
                        float(self.dim) ** -0.5, *self.states(cache.state), ctx, o, nq, floor, heads=self.heads, dim=self.dim,
                        vdim=self.vdim)
        y = torch.empty((T, vg), dtype=x.dtype, device=x.device)
        ops.head_weight_norm_gate(o, proj[:, 2 * qk + vg:], self.norm_w, self.eps, y, ctx.meta, self.heads, kind="sigmoid", nq=nq,
                                  floor=floor)
        return ops.linear(y, self.w_out, meta=ctx.meta)


register_part("mixer", "matrix_memory", MatrixMemory)
