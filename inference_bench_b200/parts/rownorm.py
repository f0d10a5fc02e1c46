"""Grouped attention whose query and key norms run over a token's whole rows, with values that may be mixed with an earlier layer's.

    q = w_q rms_unit(Wq h)  over all heads' entries at once (heads x dim),   k = w_k rms_unit(Wk h) likewise (kv_heads x dim),   v = Wv h (kv_heads x vdim)
    q and k turned by the position over the first `rotary_dim` entries of every head (entry i with i + rotary_dim/2), after the norm
    score = q . k * scale, a causal softmax, out = Wo [o_1 | o_2 | ...]
`value_mix`: None; "first": the layer's values, as projected, are what later layers of the step mix theirs with; "mix": v <- (1 - c) v + c v_first
with c a learned number of the layer and v_first the first such layer's values of the same token. The mixed values are what is cached. v_first
lives for the step (float32, `ctx.memo`): every layer sees the same tokens in a step, so nothing of it outlasts one.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from . import base
from .base import PagedKV, WeightSpec

FIRST_VALUES = "first values"   # the step memo's key of what the layers with mixed values mix with


@base.register_mixer("row_norm_attention")
class RowNormAttention(base.Mixer):
    NAMES = ("q", "k", "v", "o", "q.norm", "k.norm", "vmix")

    def __init__(self, prefix: str, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, norm_eps: float, position: base.PositionEncoding,
                 value_mix: Optional[str] = None, window: Optional[int] = None, names: tuple = NAMES):
        if heads <= 0 or kv_heads <= 0 or heads % kv_heads:
            raise ValueError(f"{heads} query heads are not a positive multiple of {kv_heads} kv heads")
        if dim <= 0 or vdim <= 0 or max(dim, vdim) > 256:
            raise ValueError(f"heads of {dim} and {vdim} must be positive and at most 256")
        if getattr(position, "pairing", "half") != "half":
            raise ValueError("this attention turns entry i with i + rotary_dim/2: it needs a position encoding with pairing=\"half\"")
        if value_mix not in (None, "first", "mix"):
            raise ValueError(f"value_mix {value_mix!r} is not known (None, first, mix)")
        self.prefix, self.hidden, self.heads, self.kv_heads, self.dim, self.vdim = prefix, hidden, heads, kv_heads, dim, vdim
        self.scale, self.norm_eps, self.position, self.value_mix, self.window, self.names = float(scale), norm_eps, position, value_mix, window, tuple(names)
        self.w_in = self.wo = self.q_norm = self.k_norm = self.mix = None

    def cache_need(self):
        row = max(self.dim, self.vdim)
        return PagedKV(self.kv_heads, row + row % 2, self.window)

    def _n(self, i: int) -> str:
        return f"{self.prefix}.{self.names[i]}"

    def weight_specs(self):
        q, k, v = self.heads * self.dim, self.kv_heads * self.dim, self.kv_heads * self.vdim
        specs = [WeightSpec(self._n(i), (n, self.hidden)) for i, n in enumerate((q, k, v))]
        specs += [WeightSpec(self._n(3), (self.hidden, self.heads * self.vdim)), WeightSpec(self._n(4), (q,), role="norm"), WeightSpec(self._n(5), (k,), role="norm")]
        return specs + ([WeightSpec(self._n(6), (), role="unit")] if self.value_mix == "mix" else [])

    def bind(self, weights, rt):
        self.w_in = rt.matrix(torch.cat([weights[self._n(i)] for i in range(3)], dim=0))   # [q | k | v]: one product
        self.wo = rt.matrix(weights[self._n(3)])
        self.q_norm, self.k_norm = rt.vector(weights[self._n(4)]), rt.vector(weights[self._n(5)])
        if self.value_mix == "mix":
            self.mix = rt.vector(weights[self._n(6)].reshape(1))
        self.position.bind(weights, rt)

    adds_to_residual = True   # the output projection may add to the residual stream in its epilogue

    def forward(self, ctx, h, cache, residual=None):
        rt, T = ctx.rt, ctx.n_tokens
        from ..kernels import attention
        cos, sin = self.position.tables(ctx)
        first = keep = None
        if self.value_mix == "first":
            keep = ctx.memo[FIRST_VALUES] = rt.empty((T, self.kv_heads * self.vdim), torch.float32)
        elif self.value_mix == "mix":
            first = ctx.memo[FIRST_VALUES]
        q = rt.empty((T, self.heads * self.dim))
        ops.row_norm_qkv(rt.linear(h, self.w_in), self.q_norm, self.k_norm, self.norm_eps, cos, sin, ctx.positions, ctx.seg_of_token, q, cache, self.heads, self.dim,
                         self.vdim, rt.status, mix=self.mix, first=first, keep=keep)
        out = attention.paged_attention(ctx, q, cache, self.heads, self.window, self.scale, qk_dim=self.dim, v_dim=self.vdim)
        return rt.linear(out, self.wo, add_to=residual)
