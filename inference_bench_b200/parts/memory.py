"""A matrix memory with exponential gates as a mixer (the mLSTM of xLSTM).

With h the layer's input, per token and head (q, k of size `dim`, v, g of size `vdim`, i and f one number each):
    q = Wq h / sqrt(dim),  k = Wk h,  v = Wv h;   i = cap tanh((Wi h + b_i) / cap),  f = logsigmoid(cap tanh((Wf h + b_f) / cap))
    m' = max(f + m, i);   S <- e^(f + m - m') S + e^(i - m') k v^T;   n <- e^(f + m - m') n + e^(i - m') k      (S, n, m zero at admission)
    o = S^T q / (max(|n . q|, e^(-m')) + 1e-6);   every head's o is divided by its root mean square over vdim;
    out = Wo ([o_1 | o_2 | ...] * w * sigmoid(Wg h)),  w a weight per channel of all heads.
All six projections are one matrix product; gates, maxima, state, o, its norm and the output gate are float32 on its float32 sums whatever the
activation dtype. n is one more column of S (a value that is always one), so the walk, the chunked form of long segments and the slots are
those of the other recurrences (parts/recurrent.py, csrc/gated_recurrence.cu).
"""
from __future__ import annotations

import torch

from ..kernels import ops
from . import base
from .base import FixedState, Several, WeightSpec
from .recurrent import GatedLinearRecurrence


@base.register_mixer("mlstm")
class MatrixMemory(base.Mixer):
    NAMES = ("q", "k", "v", "g", "i", "f", "{}.b", "norm", "o")

    def __init__(self, prefix: str, hidden: int, heads: int, dim: int, vdim: int, gate_cap: float, norm_eps: float, names: tuple = NAMES):
        if heads <= 0 or dim <= 0 or vdim <= 0 or dim > 512:
            raise ValueError(f"heads {heads}, dim {dim} (at most 512) and vdim {vdim} must be positive")
        if not gate_cap > 0:
            raise ValueError(f"the gates' cap must be positive, got {gate_cap}")
        self.prefix, self.hidden, self.heads, self.dim, self.vdim, self.cap, self.norm_eps, self.names = prefix, hidden, heads, dim, vdim, float(gate_cap), norm_eps, tuple(names)
        self.w_in = self.wo = self.i_bias = self.f_bias = self.norm_w = None

    def cache_need(self):
        return Several((FixedState((self.heads, self.dim, self.vdim + 1), torch.float32), FixedState((self.heads,), torch.float32)))

    def _n(self, i: int) -> str:
        return f"{self.prefix}.{self.names[i]}"

    def _b(self, i: int) -> str:
        return f"{self.prefix}.{self.names[6].format(self.names[i])}"

    def weight_specs(self):
        H, qk, v = self.heads, self.heads * self.dim, self.heads * self.vdim
        return [WeightSpec(self._n(i), (n, self.hidden)) for i, n in enumerate((qk, qk, v, v, H, H))] + [
            WeightSpec(self._b(4), (H,), std=0.5), WeightSpec(self._b(5), (H,), role="keep_bias"), WeightSpec(self._n(7), (v,), role="norm"),
            WeightSpec(self._n(8), (self.hidden, v))]

    def bind(self, weights, rt):
        self.w_in = rt.matrix(torch.cat([weights[self._n(i)] for i in range(6)], dim=0))     # [q | k | v | g | i | f]: one product
        self.i_bias, self.f_bias, self.norm_w = rt.vector(weights[self._b(4)]), rt.vector(weights[self._b(5)]), rt.vector(weights[self._n(7)])
        self.wo = rt.matrix(weights[self._n(8)])

    adds_to_residual = True   # the output projection may add to the residual stream in its epilogue

    def forward(self, ctx, h, cache, residual=None):
        rt, H, D, V = ctx.rt, self.heads, self.dim, self.vdim
        state, m_state = cache
        proj = rt.linear(h, self.w_in)
        cols, at = [], 0
        for n in (H * D, H * D, H * V, H * V, H, H):
            cols.append(ops.Parts.columns(proj, at))
            at += n
        out = rt.empty((ctx.n_tokens, H * V))
        short, long_segs, chunks = GatedLinearRecurrence._cut(ctx)
        ops.memory_recurrence(*cols, self.i_bias, self.f_bias, self.cap, state.tensor, m_state.tensor, ctx.seg_start, ctx.seg_slot, ctx.n_segments, self.norm_w,
                              self.norm_eps, out, H, D, V, single_tokens=ctx.fixed_shape or ctx.n_segments == ctx.n_tokens, seg_list=short, long_segs=long_segs, chunks=chunks)
        return rt.linear(out, self.wo, add_to=residual)
