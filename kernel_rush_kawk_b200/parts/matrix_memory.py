"""Mixers with a matrix state per head whose key and value sizes differ, written without a removal term.

Per head S is N x P (``dim`` x ``vdim``), 32-bit, zero at the start of a sequence and carried from token to token;
q = Wq h / sqrt(N), k = Wk h, v = Wv h.

* ``GatedLinearAttention`` (kind "gla"): row n of S decays by alpha_n = exp(logsigmoid(z_n) / tau), z = Wa2 (Wa1 h) + b;
  S <- diag(alpha) S + k v^T, o = S^T q. The readout of every head passes an RMS norm whose weight (P numbers) is one for
  all heads; then silu(Wg h) times that, side by side, is projected.
* ``MatrixLSTM`` (kind "mlstm"): with c(x) = cap tanh(x / cap), a head's log gates are i = c(Wi h + bi) for the input and
  f = logsigmoid(c(Wf h + bf)) for what is kept. With a running maximum m (zero at the start), m' = max(f + m, i):
  S <- exp(f + m - m') S + exp(i - m') k v^T, n <- exp(f + m - m') n + exp(i - m') k,
  o = S^T q / (max(|n . q|, exp(-m')) + 1e-6). o over its own root mean square, head by head, meets a weight over all
  heads' columns and sigmoid(Wg h), and is projected. n and m are state as well.

Gates, decays, the state and o are 32-bit on every path; the projections run in the path's dtype. All projections of h
ride in one stacked product.
"""

from __future__ import annotations

import torch

from .base import StateNeed, TensorSpec, register_mixer
from .branches import Branch


class _MatrixMemory(Branch):
    def __init__(self, params):
        super().__init__(params)
        p = params
        self.hidden = int(p["hidden"])
        self.heads = int(p["heads"])
        self.dim = int(p["dim"])
        self.vdim = int(p["vdim"])
        self.eps = float(p["eps"])
        self.keys, self.values = self.heads * self.dim, self.heads * self.vdim

    def tensor_specs(self):
        C, HN, HP = self.hidden, self.keys, self.values
        return {"q": TensorSpec((HN, C)), "k": TensorSpec((HN, C)), "v": TensorSpec((HP, C)), "g": TensorSpec((HP, C)),
                "o": TensorSpec((C, HP))}

    def out_weight(self):
        return self.w["o"]

    def in_weight(self):
        return torch.cat([self.w[k] for k in ("q", "k", "v", "g") + self.EXTRA], dim=0)

    def _columns(self, proj):
        """q, k, v, gate and the rest as column slices of the stacked product."""
        HN, HP = self.keys, self.values
        return (proj[:, :HN], proj[:, HN:2 * HN], proj[:, 2 * HN:2 * HN + HP], proj[:, 2 * HN + HP:2 * (HN + HP)],
                proj[:, 2 * (HN + HP):])


class GatedLinearAttention(_MatrixMemory):
    """params: hidden, heads, dim, vdim, rank, tau, eps."""

    EXTRA = ("a1",)

    def __init__(self, params):
        super().__init__(params)
        self.rank = int(params["rank"])
        self.tau = float(params["tau"])

    def tensor_specs(self):
        specs = super().tensor_specs()
        specs.update({"a1": TensorSpec((self.rank, self.hidden)), "a2": TensorSpec((self.keys, self.rank)),
                      "a2.b": TensorSpec((self.keys,), "vector"), "norm": TensorSpec((self.vdim,), "gain")})
        return specs

    def cache_need(self):
        return StateNeed((self.heads, self.dim, self.vdim), "float32")

    def bind(self, tensors, runtime):
        self.w = dict(tensors)
        self.a2 = tensors["a2"].contiguous()
        self.a2_bias = tensors["a2.b"].float().contiguous()
        self.norm_w = tensors["norm"].float().contiguous()
        self.bind_standalone()

    def middle(self, ctx, proj, cache, out, col0, scale):
        q, k, v, g, rest = self._columns(proj)
        ctx.ops.gla_scan(q, k, v, g, rest[:, :self.rank], self.a2, self.a2_bias, self.tau, self.heads, self.dim, self.vdim,
                         self.norm_w, self.eps, cache.state, ctx.batch, out, col0, scale)


class MatrixLSTM(_MatrixMemory):
    """params: hidden, heads, dim, vdim, gate_cap, eps."""

    EXTRA = ("i", "f")

    def __init__(self, params):
        super().__init__(params)
        self.cap = float(params["gate_cap"])

    def tensor_specs(self):
        specs = super().tensor_specs()
        H = self.heads
        specs.update({"i": TensorSpec((H, self.hidden)), "i.b": TensorSpec((H,), "vector"),
                      "f": TensorSpec((H, self.hidden)), "f.b": TensorSpec((H,), "vector"),
                      "norm": TensorSpec((self.values,), "gain")})
        return specs

    def cache_need(self):
        # the matrix; then n and, behind it, m
        return (StateNeed((self.heads, self.dim, self.vdim), "float32"), StateNeed((self.heads, self.dim + 1), "float32"))

    def bind(self, tensors, runtime):
        self.w = dict(tensors)
        self.gate_bias = torch.cat([tensors["i.b"].float(), tensors["f.b"].float()]).contiguous()
        self.norm_w = tensors["norm"].float().contiguous()
        self.bind_standalone()

    def middle(self, ctx, proj, cache, out, col0, scale):
        q, k, v, g, rest = self._columns(proj)
        ctx.ops.mlstm_scan(q, k, v, g, rest[:, :2 * self.heads], self.gate_bias, self.cap, self.heads, self.dim, self.vdim,
                           self.norm_w, self.eps, cache[0].state, cache[1].state, ctx.batch, out, col0, scale)


register_mixer("gla", GatedLinearAttention)
register_mixer("mlstm", MatrixLSTM)
