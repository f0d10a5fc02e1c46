"""A feed-forward of routed experts: every token runs through a few of many small gated feed-forwards, chosen by a router,
plus (optionally) one shared expert that every token uses.

    s = softmax(Wr h) over all experts (float32);  experts lie in `groups` equal groups of neighbours, a group's score is its
    largest s, the best `groups_keep` groups stay;  of their experts the `top` with the largest s are chosen;
    out = sum_e weight_e * down_e(silu(gate_e h) * up_e h)  [+ shared(h)],   weight_e = s_e * route_scale
    (with `renorm`: s_e / sum of the chosen s, times route_scale).
`score="sigmoid"`: s_e = sigmoid of expert e's own logit instead of the softmax. `correction` names a tensor of one number an expert
that is added to s where groups and experts are chosen and left out of the weights; `group_top` n makes a group's score the sum of
its n largest choice scores (experts of groups that do not stay cannot be chosen, whatever the sign of their scores). `weight_on="input"`: the weight scales what the expert
reads, out = sum_e down_e(silu(gate_e (weight_e h)) * up_e (weight_e h)), which is not the same thing for a gated expert.
`score="chosen_softmax"`: the `top` experts with the largest logits are chosen and weighted by the softmax over the chosen logits alone;
`router_bias` names a bias of the logits. `activation="relu2"`: experts and shared expert without a gate, down_e(max(up_e h, 0)^2).
`activation="clamped_swiglu"` with clamp = (limit, slope): gated with clamped halves, g sigmoid(slope g) (u + 1) with g = min(gate, limit) and
u = up cut to [-limit, limit]; the shared expert has a limit of its own (`shared_limit`).
`shared_gate` names a vector (one row): the shared expert's output is multiplied by the sigmoid of its product with the token's row.
The step's (token, expert) pairs are regrouped by expert on the device (no trip to the host, so the step can be captured),
the experts' products run on the regrouped rows, and the weighted sum returns them to token order.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..kernels import gemm_tcgen05 as G
from ..kernels import ops
from . import base
from .base import WeightSpec


FEW_TOKENS = 64         # up to here the shared expert runs beside the routed ones
ROUTE_SORT_TOKENS = 32  # up to here the choice and the regrouping are one kernel (a warp of one CTA per token)


@base.register_feed_forward("routed_experts")
class RoutedExperts(base.FeedForward):
    def __init__(self, prefix: str, hidden: int, expert_ff: int, experts: int, top: int, route_scale: float = 1.0, groups: int = 1, groups_keep: int = 1,
                 shared_ff: int = 0, renorm: bool = False, names: tuple = ("router", "e{}", "shared", "gate", "up", "down"), score: str = "softmax",
                 weight_on: str = "output", correction: str = "", group_top: int = 1, activation: str = "swiglu", router_bias: str = "", shared_gate: str = "",
                 clamp: Optional[tuple] = None, shared_limit: float = 0.0):
        if not 0 < top <= experts or experts % groups or not 0 < groups_keep <= groups:
            raise ValueError(f"top {top} of {experts} experts in {groups} groups of which {groups_keep} stay")
        if activation not in ("swiglu", "relu2", "clamped_swiglu"):
            raise ValueError(f"activation {activation!r} is not known (swiglu, relu2, clamped_swiglu)")
        if (clamp is not None) != (activation == "clamped_swiglu") or (clamp is not None and (not clamp[0] > 0 or (shared_ff and not shared_limit > 0))):
            raise ValueError("the clamped activation, and no other, takes clamp = (limit, slope), and with a shared expert a limit for it")
        self.gated, self.router_bias, self.shared_gate = activation != "relu2", router_bias, shared_gate if shared_ff else ""
        self.clamp, self.shared_limit = clamp, float(shared_limit)
        self.limits = self.shared_clamp = None      # `ops.Clamp` of the experts (then the shared expert's blocks), and of the shared expert alone
        self.b_router, self.blocks = None, 0
        if score not in ops.ROUTE_SCORES or weight_on not in ("output", "input"):
            raise ValueError(f"score {score!r} ({', '.join(ops.ROUTE_SCORES)}) or weight_on {weight_on!r} (output, input) is not known")
        if not 1 <= group_top <= 4:
            raise ValueError(f"a group's score is the sum of its {group_top} largest scores: 1 to 4 are built")
        self.score, self.weight_on, self.correction, self.group_top = score, weight_on, correction, int(group_top)
        self.w_correction = None
        self.prefix, self.hidden, self.expert_ff, self.experts, self.top = prefix, hidden, expert_ff, experts, top
        self.route_scale, self.groups, self.groups_keep, self.shared_ff, self.renorm, self.names = route_scale, groups, groups_keep, shared_ff, renorm, tuple(names)
        self.w_router = self.w_gu = self.w_d = self.shared_gu = self.shared_d = None

    def _expert(self, k: int, which: int) -> str:
        return f"{self.prefix}.{self.names[1].format(k)}.{self.names[3 + which]}"

    def _shared(self, which: int) -> str:
        return f"{self.prefix}.{self.names[2]}.{self.names[3 + which]}"

    def weight_specs(self):
        W, F = self.hidden, self.expert_ff
        specs = [WeightSpec(f"{self.prefix}.{self.names[0]}", (self.experts, W))]
        gate = (0,) if self.gated else ()
        for k in range(self.experts):
            specs += [WeightSpec(self._expert(k, i), (F, W)) for i in (*gate, 1)] + [WeightSpec(self._expert(k, 2), (W, F))]
        if self.router_bias:
            specs.append(WeightSpec(f"{self.prefix}.{self.router_bias}", (self.experts,), std=0.1))
        if self.correction:
            specs.append(WeightSpec(f"{self.prefix}.{self.correction}", (self.experts,), std=0.1))
        if self.shared_ff:
            S = self.shared_ff
            specs += [WeightSpec(self._shared(i), (S, W)) for i in (*gate, 1)] + [WeightSpec(self._shared(2), (W, S))]
            if self.shared_gate:
                specs.append(WeightSpec(f"{self.prefix}.{self.names[2]}.{self.shared_gate}", (1, W)))
        return specs

    def bind(self, weights, rt):
        router = weights[f"{self.prefix}.{self.names[0]}"]
        if self.shared_gate:   # the shared expert's gate is one more row of the router's product
            router = torch.cat([router, weights[f"{self.prefix}.{self.names[2]}.{self.shared_gate}"]], dim=0)
        self.w_router = rt.matrix(router)
        if self.router_bias:
            self.b_router = rt.vector(weights[f"{self.prefix}.{self.router_bias}"])
        if self.correction:
            self.w_correction = rt.vector(weights[f"{self.prefix}.{self.correction}"])
        # [experts, gate rows then up rows, width] and [experts, width, inner]: one tensor each, so a tile of the grouped product finds its expert by an offset
        front = (0, 1) if self.gated else (1,)
        S, F = self.shared_ff, self.expert_ff
        self.blocks = S // F if S and S % F == 0 and (not self.gated or self.clamp is not None) and self.weight_on == "output" else 0
        gu = [torch.cat([weights[self._expert(k, i)] for i in front], dim=0) for k in range(self.experts)]
        down = [weights[self._expert(k, 2)] for k in range(self.experts)]
        if S:
            shared_gu, shared_d = torch.cat([weights[self._shared(i)] for i in front], dim=0), weights[self._shared(2)]
            # the shared expert's inner channels in blocks of a routed expert's size, behind the routed experts
            if self.blocks and self.gated:
                gate, up = shared_gu.split(S)
                gu += [torch.cat([gate[b:b + F], up[b:b + F]], dim=0) for b in range(0, S, F)]
            elif self.blocks:
                gu += list(shared_gu.split(F))
            down += list(shared_d.split(F, dim=1)) if self.blocks else []
        self.w_gu, self.w_d = rt.upload(torch.stack(gu), rt.act_dtype), rt.upload(torch.stack(down), rt.act_dtype)
        if S:
            # (a view where the blocks hold it as it is: a gated one in several blocks has its gate and up rows elsewhere)
            whole = self.blocks and (not self.gated or self.blocks == 1)
            self.shared_gu = rt.matrix(self.w_gu[self.experts:].reshape(-1, self.hidden) if whole else shared_gu)
            self.shared_d = rt.matrix(self.w_d[self.experts] if self.blocks == 1 else shared_d)
        if self.clamp is not None:
            limit, slope = self.clamp
            self.limits = ops.Clamp(rt.upload(torch.tensor([limit] * self.experts + [self.shared_limit] * self.blocks, dtype=torch.float32)), slope)
            if S:
                self.shared_clamp = ops.Clamp(rt.upload(torch.tensor([self.shared_limit], dtype=torch.float32)), slope)

    def forward(self, ctx, h):
        rt, T, E, top = ctx.rt, ctx.n_tokens, self.experts, self.top
        logits = rt.linear(h, self.w_router)                     # float32 partial sums [P, T, E (+ 1)]
        # few tokens: a shared expert that is whole blocks of the routed experts' size runs as further experts that every token uses (in float32
        # always, so that a token's sums run in one order however many share its step)
        always = self.blocks if T <= FEW_TOKENS or rt.act_dtype == torch.float32 else 0
        n, used = E + always, top + always
        R = T * used
        idx, wt = rt.empty((T, used), torch.int32), rt.empty((T, used), torch.float32)
        on_input = self.weight_on == "input"
        offsets, tile_start = rt.empty((n + 1,), torch.int32), rt.empty((n + 1,), torch.int32)
        row_of_pair, token_of_row = rt.empty((R,), torch.int32), rt.empty((R,), torch.int32)
        how = rt.options.expert_gemm
        bn = G.grouped_token_tile(R, n, self.expert_ff, rt.sm_count)
        act = rt.empty((R, self.expert_ff))
        y = rt.empty((R, self.hidden), torch.float32)
        tcgen05 = how in ("auto", "tcgen05") and rt.act_dtype == torch.bfloat16 and rt.gemm != "simt" and G.grouped_supported(self.hidden, self.expert_ff, bn, self.gated)
        if how == "tcgen05" and not tcgen05:
            raise ValueError(f"expert_gemm = \"tcgen05\" needs bfloat16 and inner sizes that are multiples of 8 (of 64 for few tokens), got {self.hidden} and {self.expert_ff}")
        tile_rows = bn if tcgen05 else ops.moe_tile_rows()
        one = T <= ROUTE_SORT_TOKENS and ops.moe_route_sort_fits(T, E, self.groups, always)     # the choice and the regrouping in one kernel
        ops.moe_route(logits, self.groups, self.groups_keep, top, self.route_scale, self.renorm, idx, wt, self.score, correction=self.w_correction, group_top=self.group_top,
                      experts=E, logit_bias=self.b_router, always=always, gate_col=E if self.shared_gate and always else -1,
                      sort=(offsets, tile_start, row_of_pair, token_of_row, tile_rows) if one else None)
        if not one:
            ops.moe_sort(idx, n, offsets, tile_start, row_of_pair, token_of_row, tile_rows=tile_rows)
        w_gu, w_d = self.w_gu[:n], self.w_d[:n]
        if tcgen05:   # the tcgen05 kernel of the single-matrix products, its tiles taking their expert from the tile table
            xs = rt.empty((R, self.hidden))
            if on_input:
                ops.scatter_scaled_rows(h, row_of_pair, wt, xs)
            else:
                ops.gather_rows(h, token_of_row, xs)
            if self.gated:
                G.gemm_grouped_swiglu(xs, w_gu, act, bn, offsets, tile_start, rt.status, clamp=self.limits)
            else:
                G.gemm_grouped_relu2(xs, w_gu, act, bn, offsets, tile_start, rt.status)
            G.gemm_grouped(act, w_d, y, bn, offsets, tile_start, rt.status)
        else:
            tc = how != "simt"
            src, rows = h, token_of_row
            if on_input:   # the rows in the experts' order, each times its weight; the product then reads them as they lie
                src, rows = rt.empty((R, self.hidden)), None
                ops.scatter_scaled_rows(h, row_of_pair, wt, src)
            ops.gemm_grouped(src, rows, w_gu, act, offsets, tile_start, gated=self.gated, tensor_cores=tc and ops.rows_mma_fits(src, w_gu),
                             act="none" if self.gated else "relu2", clamp=self.limits)
            ops.gemm_grouped(act, None, w_d, y, offsets, tile_start, gated=False, tensor_cores=tc and ops.rows_mma_fits(act, w_d))
        shared = None
        if self.shared_ff and not always:
            shared = rt.linear(rt.gate_up_act(h, self.shared_gu, self.shared_clamp) if self.gated else rt.up_act(h, self.shared_gu, "relu2"), self.shared_d)
        out = rt.empty((1, T, self.hidden), torch.float32)
        ops.moe_combine(y, row_of_pair, wt, shared, out[0], weighted=not on_input, gate=(logits, E) if self.shared_gate and shared is not None else None)
        return out
