"""Differential attention: a head scores every key twice, with two maps of its query and key, and subtracts the second softmax's output.

    q = Wq h + bq  (heads x 2 x dim),  k = Wk h + bk  (kv_heads x 2 x dim),  v = Wv h + bv  (kv_heads x vdim)
    every map of q and k is turned by the position over its first `rotary_dim` entries
    a_m = softmax over the visible keys of (q_m . k_m) * scale, times v   (m = 1, 2; both over the same v)
    u = a_1 - lambda a_2,   lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff   (one number a layer, made when the weights are loaded)
    out = Wo [(1 - diff) u / sqrt(mean(u^2) + eps), per head]
A position sees itself and the `window` - 1 before it, and with `keep_first` n also the positions 0 .. n - 1. With `own_kv` False the
layer has no key and value projections: it reads the cache of another execution, whose heads and rotation are the same.

The cache holds a key row of both maps and a value row per kv head. A query is written once per map as a row of a key's width with zeros
outside the map's part (csrc/diff_attention.cu), so every attention kernel of the engine serves the design as 2 x heads query heads: with
2 dim = vdim of 64 or 128 in bfloat16 the tensor-core kernels (prompt portions and decoded tokens), anything else the generic kernel.
"""
from __future__ import annotations

import math
from typing import Optional

import torch

from ..kernels import ops
from . import base
from .base import PagedKV, WeightSpec

MAPS = 2


@base.register_mixer("differential_attention")
class DifferentialAttention(base.Mixer):
    NAMES = ("q", "k", "v", "o", "{}.b", "lq1", "lk1", "lq2", "lk2")

    def __init__(self, prefix: str, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, diff: float, norm_eps: float,
                 position: base.PositionEncoding, window: Optional[int] = None, keep_first: int = 0, own_kv: bool = True, cache_window: Optional[int] = -1,
                 cache_keep: Optional[int] = None, names: tuple = NAMES):
        """cache_window, cache_keep: what the cache has to hold when other executions read it too (default: this layer's own window and first
        positions; cache_window None: everything)."""
        if heads <= 0 or kv_heads <= 0 or heads % kv_heads:
            raise ValueError(f"{heads} query heads are not a positive multiple of {kv_heads} kv heads")
        if dim <= 0 or vdim <= 0 or max(MAPS * dim, vdim) > 256:
            raise ValueError(f"two maps of {dim} and values of {vdim} must be positive and at most 256")
        self.prefix, self.hidden, self.heads, self.kv_heads, self.dim, self.vdim = prefix, hidden, heads, kv_heads, dim, vdim
        self.scale, self.diff, self.norm_eps, self.position = float(scale), float(diff), norm_eps, position
        self.window, self.keep_first, self.own_kv, self.names = window, int(keep_first), own_kv, tuple(names)
        self.cache_window = window if cache_window == -1 else cache_window
        self.cache_keep = self.keep_first if cache_keep is None else int(cache_keep)
        self.w_in = self.in_bias = self.wo = self.lam = None

    def cache_need(self):
        row = max(MAPS * self.dim, self.vdim)
        return PagedKV(self.kv_heads, row + row % 2, self.cache_window, self.cache_keep if self.cache_window else 0) if self.own_kv else None

    def _n(self, i: int) -> str:
        return f"{self.prefix}.{self.names[i]}"

    def _b(self, i: int) -> str:
        return f"{self.prefix}.{self.names[4].format(self.names[i])}"

    def weight_specs(self):
        rows = [self.heads * MAPS * self.dim, self.kv_heads * MAPS * self.dim, self.kv_heads * self.vdim]
        own = range(3) if self.own_kv else range(1)
        specs = [WeightSpec(self._n(i), (rows[i], self.hidden)) for i in own] + [WeightSpec(self._b(i), (rows[i],), std=0.1) for i in own]
        specs += [WeightSpec(self._n(i), (self.dim,), std=0.1) for i in range(5, 9)]
        return specs + [WeightSpec(self._n(3), (self.hidden, self.heads * self.vdim))]

    def bind(self, weights, rt):
        own = range(3) if self.own_kv else range(1)
        self.w_in = rt.matrix(torch.cat([weights[self._n(i)] for i in own], dim=0))
        self.in_bias = rt.vector(torch.cat([weights[self._b(i)].to(torch.float32) for i in own]))
        lq1, lk1, lq2, lk2 = (weights[self._n(i)].to("cpu", torch.float32) for i in range(5, 9))
        self.lam = math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + self.diff
        self.wo = rt.matrix(weights[self._n(3)])
        self.position.bind(weights, rt)

    def forward(self, ctx, h, cache):
        rt, T = ctx.rt, ctx.n_tokens
        from ..kernels import attention
        cos, sin = self.position.tables(ctx)
        q = rt.empty((T, self.heads * MAPS * MAPS * self.dim))
        ops.map_qkv(rt.linear(h, self.w_in), self.in_bias, cos, sin, getattr(self.position, "pairing", "half") == "interleaved", ctx.positions, ctx.seg_of_token, q, cache,
                    self.heads, MAPS, self.dim, self.vdim, rt.status, write_kv=self.own_kv)
        out = attention.paged_attention(ctx, q, cache, self.heads * MAPS, self.window, self.scale, qk_dim=MAPS * self.dim, v_dim=self.vdim, keep_first=self.keep_first,
                                        diff=(self.lam, self.norm_eps, 1.0 - self.diff))
        return rt.linear(out, self.wo)
