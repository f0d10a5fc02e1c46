"""Linear recurrences whose queries, keys and values are plain projections: a fixed decay per head (retention), and a decay per channel
and token behind a token shift, with a bonus for the current token (the RWKV time mix).

"retention":  q = Wq h, k = Wk h (heads x dim), v = Wv h (heads x vdim); q and k turned by the position over their first `rotary_dim` entries, k
    times dim^(-1/2) after that;  S <- decay_head S + k v^T,  o = S^T q;  o goes through a weightless RMS norm per head, is gated by silu(Wg h) and projected.

"wkv":  every one of r, k, v, g, w reads a mix of its own, h + (h' - h) mu, with h' the previous token's normed row (zeros before the first);
    w = exp(-exp(W2 tanh(W1 mix_w) + w0));  o = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T;  o goes through an RMS norm per head
    with a weight per channel of all heads, is gated by silu(Wg mix_g) and projected.

State (S, and the last normed row) is float32 and lives in the request's slot; rotation, decays, gates, o and its norm are float32 on the
products' float32 sums, whatever the activation dtype. The walk is the recurrence kernel of csrc/gated_recurrence.cu: segments of more than
`ops.RECURRENCE_CHUNK` tokens go through its chunked form, by their own length only (parts/recurrent.py).

The five mixes are made where the rows are normed: the mixer runs its input norm itself (`runs_norm`), for a step of single tokens in one
kernel with the residual add, the norm and the state (csrc/layernorm.cu).
"""
from __future__ import annotations

import math

import torch

from ..kernels import gemm_tcgen05 as G
from ..kernels import ops
from . import base
from .base import FixedState, Several, WeightSpec
from .recurrent import GatedLinearRecurrence


@base.register_mixer("retention")
class Retention(base.Mixer):
    NAMES = ("q", "k", "v", "g", "o")

    def __init__(self, prefix: str, hidden: int, heads: int, dim: int, vdim: int, decay, norm_eps: float, position: base.PositionEncoding, names: tuple = NAMES):
        decay = tuple(float(x) for x in decay)
        if heads <= 0 or dim <= 0 or vdim <= 0 or dim > 512:
            raise ValueError(f"heads {heads}, dim {dim} (at most 512) and vdim {vdim} must be positive")
        if len(decay) != heads or any(not 0.0 <= x <= 1.0 for x in decay):
            raise ValueError(f"{heads} heads need {heads} decays in [0, 1], got {decay}")
        if getattr(position, "pairing", "half") != "half":
            raise ValueError("this mixer turns entry i with i + rotary_dim/2: it needs a position encoding with pairing=\"half\"")
        self.prefix, self.hidden, self.heads, self.dim, self.vdim, self.decay = prefix, hidden, heads, dim, vdim, decay
        self.norm_eps, self.position, self.names = norm_eps, position, tuple(names)
        self.w_in = self.wo = self.decay_dev = None

    def cache_need(self):
        return FixedState((self.heads, self.dim, self.vdim), torch.float32)

    def _n(self, i: int) -> str:
        return f"{self.prefix}.{self.names[i]}"

    def weight_specs(self):
        qk, v = self.heads * self.dim, self.heads * self.vdim
        return [WeightSpec(self._n(i), (n, self.hidden)) for i, n in enumerate((qk, qk, v, v))] + [WeightSpec(self._n(4), (self.hidden, v))]

    def bind(self, weights, rt):
        self.w_in = rt.matrix(torch.cat([weights[self._n(i)] for i in range(4)], dim=0))     # [q | k | v | g]: one product
        self.wo = rt.matrix(weights[self._n(4)])
        self.decay_dev = rt.upload(torch.tensor(self.decay, dtype=torch.float32))
        self.position.bind(weights, rt)

    def forward(self, ctx, h, cache):
        rt, T, H, D, V = ctx.rt, ctx.n_tokens, self.heads, self.dim, self.vdim
        cos, sin = self.position.tables(ctx)
        proj = rt.linear(h, self.w_in)
        o = rt.empty((T, H, V), torch.float32)
        short, long_segs, chunks = GatedLinearRecurrence._cut(ctx)
        part = lambda col: ops.Parts.columns(proj, col)
        ops.recurrence("turned", part(0), part(H * D), part(2 * H * D), self.decay_dev, cache.tensor, ctx.seg_start, ctx.seg_slot, ctx.n_segments, o, H, D, V, seg_list=short,
                       long_segs=long_segs, chunks=chunks, cos=cos, sin=sin, k_scale=1.0 / math.sqrt(D))
        out = rt.empty((T, H * V))
        ops.head_norm_gate(o, None, self.norm_eps, part(2 * H * D + H * V), out)
        return rt.linear(out, self.wo)


@base.register_mixer("wkv")
class WkvMixer(base.Mixer):
    runs_norm = True
    MIXES = ("r", "k", "v", "g", "w")
    NAMES = ("mu.{}", "r", "k", "v", "g", "w1", "w2", "w0", "u", "norm", "o")

    def __init__(self, prefix: str, hidden: int, heads: int, dim: int, norm_eps: float, decay_rank: int = 64, names: tuple = NAMES):
        """decay_rank: the inner size of the decay's two matrices for random weights; a checkpoint's own tensors decide it otherwise."""
        if heads <= 0 or dim <= 0 or dim > 512:
            raise ValueError(f"heads {heads} and dim {dim} (at most 512) must be positive")
        self.prefix, self.hidden, self.heads, self.dim, self.norm_eps, self.decay_rank, self.names = prefix, hidden, heads, dim, norm_eps, int(decay_rank), tuple(names)
        self.mu = self.w_rkvg = self.stacked = self.w1 = self.w2 = self.w0 = self.u = self.norm_w = self.wo = None

    def cache_need(self):
        return Several((FixedState((self.heads, self.dim, self.dim), torch.float32), FixedState((self.hidden,), torch.float32)))

    def _n(self, i: int) -> str:
        return f"{self.prefix}.{self.names[i]}"

    def _mu(self, s: str) -> str:
        return f"{self.prefix}.{self.names[0].format(s)}"

    def weight_specs(self):
        C, W = self.heads * self.dim, self.hidden
        return [WeightSpec(self._mu(s), (W,), role="unit") for s in self.MIXES] + [WeightSpec(self._n(i), (C, W)) for i in range(1, 5)] + [
            WeightSpec(self._n(5), (self.decay_rank, W), free=(0,)), WeightSpec(self._n(6), (C, self.decay_rank), free=(1,)), WeightSpec(self._n(7), (C,), role="decay_bias"),
            WeightSpec(self._n(8), (self.heads, self.dim), std=0.5), WeightSpec(self._n(9), (C,), role="norm"), WeightSpec(self._n(10), (W, C))]

    def bind(self, weights, rt):
        self.mu = rt.vector(torch.stack([weights[self._mu(s)] for s in self.MIXES]))                      # [5, W], in the order of MIXES
        self.stacked = rt.upload(torch.stack([weights[self._n(i)] for i in range(1, 5)]), rt.act_dtype)      # [4, C, W]: r, k, v, g
        self.w_rkvg = [rt.matrix(w) for w in self.stacked]
        w1, w2 = weights[self._n(5)], weights[self._n(6)]
        if w1.shape[0] != w2.shape[1]:
            raise ValueError(f"{self._n(5)} has {w1.shape[0]} rows, {self._n(6)} has {w2.shape[1]} columns")
        self.w1 = rt.matrix(w1)
        self.w2 = rt.vector(w2.t().contiguous())                                                        # [rank, C]
        self.w0, self.u, self.norm_w = rt.vector(weights[self._n(7)]), rt.vector(weights[self._n(8)].reshape(-1)), rt.vector(weights[self._n(9)])
        self.wo = rt.matrix(weights[self._n(10)])

    def forward_normed(self, ctx, norm, x, pending, cache):
        rt, T, M = ctx.rt, ctx.n_tokens, len(self.MIXES)
        state, last = cache
        mixes = rt.empty((M, T, self.hidden))
        norm.forward_mixes(ctx, x, pending, self.mu, last.tensor, mixes)
        return self._mix(ctx, mixes, state)

    def _mix(self, ctx, mixes, state):
        rt, T, H, D = ctx.rt, ctx.n_tokens, self.heads, self.dim
        if T <= G.PARTS_MAX_TOKENS and rt.mode == "bfloat16" and rt.gemm != "simt" and G.supports(self.hidden):   # few tokens: the four products as one launch
            z = G.gemm_parts(rt, mixes[:4], self.stacked)
            r, k, v, g = (ops.Parts(z, z.shape[0], 4 * T * H * D, H * D, i * T * H * D) for i in range(4))
        else:
            r, k, v, g = (ops.Parts.columns(rt.linear(mixes[i], w)) for i, w in enumerate(self.w_rkvg))
        decay = rt.empty((T, H * D), torch.float32)
        ops.decay_rows(rt.linear(mixes[4], self.w1), self.w2, self.w0, decay)
        o = rt.empty((T, H, D), torch.float32)
        short, long_segs, chunks = GatedLinearRecurrence._cut(ctx)
        ops.recurrence("bonus", r, k, v, self.u, state.tensor, ctx.seg_start, ctx.seg_slot, ctx.n_segments, o, H, D, D, seg_list=short, long_segs=long_segs, chunks=chunks, decay=decay)
        out = rt.empty((T, H * D))
        ops.head_norm_gate(o, self.norm_w, self.norm_eps, g, out)
        return rt.linear(out, self.wo)
