"""Fedipel in the engine against the plain implementation: each mechanism's kernels alone (with weights or inputs made so that a key just
inside or just outside a window, a kept first position, a far key or a lost state row shows), then whole models under every way of cutting the
work (in true 32-bit and in bfloat16), pages and slots that are used again, and greedy generation through the engine's entry point and
scheduler."""
from __future__ import annotations

import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_fedipel as P
import tiny_fedipel as tf
import traces

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
TOLERANCE = {"float32": 1e-4, "bfloat16": 5e-2}   # of the largest |logit| of the sequence
BF16_MEDIAN = 1.5e-2


@pytest.fixture(scope="module")
def rt16():
    from inference_bench_b200.engine.runtime import Runtime
    return Runtime(DEV, dtype="bfloat16")


@pytest.fixture(scope="module")
def rt32():
    from inference_bench_b200.engine.runtime import Runtime
    return Runtime(DEV, dtype="float32")


@pytest.fixture(scope="module")
def fdirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("fedipel")
    return {name: tf.write_model(name, root / name) for name in tf.CONFIGS}


def _f32(t):
    return t.to(DEV, torch.float32).contiguous()


def _ctx(rt, runs, slots=None):
    """A step's context for segments given as (first position, tokens)."""
    from inference_bench_b200.engine.context import Segment, build_context
    return build_context(rt, [Segment(i, (slots[i] if slots else i), p0, [0] * n, []) for i, (p0, n) in enumerate(runs)])


def _steps(rt, plan, slot, reused, zero_slot, step_fn):
    """Runs a plan of [(request, tokens), ...] steps: requests in the given slots; `reused` takes a slot that another request had."""
    at = {}
    for step in plan:
        for r, _ in step:
            if r in reused and r not in at:
                zero_slot(slot[r])
            at.setdefault(r, 0)
        step_fn(_ctx(rt, [(at[r], n) for r, n in step], [slot[r] for r, _ in step]), step, dict(at))
        for r, n in step:
            at[r] += n


SHORT = [[("a", 1), ("b", 2)], [("a", 1), ("b", 1)], [("a", 2)], [("a", 7), ("b", 6)], [("c", 1), ("a", 3)], [("c", 2), ("a", 9)], [("c", 11)], [("c", 1)], [("c", 1)]]


def _long(C):
    return [[("a", 2 * C + 2), ("b", 3)], [("a", 1), ("b", C + 1)], [("a", 3 * C), ("b", 1)], [("c", C), ("a", 1)], [("c", 4 * C - 1), ("a", C + 7)], [("c", 1)]]


SLOTS = {"a": 0, "b": 1, "c": 1}      # b ends before c begins; c takes its slot, zeroed


def _lens(plan):
    lens = {}
    for step in plan:
        for r, n in step:
            lens[r] = lens.get(r, 0) + n
    return lens


# ------------------------------------------------------------------------------------------ attention over a window and the first positions
def _kept_case(rt, dtype, heads, kv_heads, dim, page, window, keep, tol):
    """Prompt portions across window, page and tile edges, the first tokens of a sequence, and single decoded tokens, all of one request on
    shuffled pages; pages that nobody can see are missing from the block table. Keys stand out for a query (they share a large entry): the
    last position of its window, the one before it, the last kept position, the first that is not kept."""
    from inference_bench_b200.kernels import attention
    from inference_bench_b200.kernels.ops import KvLayerView
    n_ctx, scale = 420, 0.35
    g = torch.Generator().manual_seed(heads * dim + page + window + keep)
    runs = [(0, 7), (130, 150), (410, 1), (window + keep, 1), (window + keep + 1, 1), (2 * page - 2, 4), (330, 70), (300, 1), (min(keep, 400), 1), (419, 1)]
    runs = [(p0, n) for p0, n in runs if p0 + n <= n_ctx]
    positions = [p0 + i for p0, n in runs for i in range(n)]
    T = len(positions)
    n_pages = -(-n_ctx // page)
    perm = torch.randperm(n_pages + 3, generator=g)[:n_pages]
    k, v = torch.randn((n_ctx, kv_heads, dim), generator=g), torch.randn((n_ctx, kv_heads, dim), generator=g)
    q = torch.randn((n_ctx, heads, dim), generator=g) * 0.3
    needles = [(410, 410 - window + 1, 0), (419, 419 - window, 1 % heads), (300, keep - 1, 2 % heads), (399, keep, 0), (398, 398 - window + 1, 1 % heads),
               (397, 397 - window, 2 % heads), (396, keep - 1, 0), (395, 0, 1 % heads), (270, 270 - window, 0), (269, keep, 1 % heads), (6, 0, 0), (131, 131, 1 % heads)]
    for i, (qp, key, head) in enumerate(needles):
        if 0 <= key < n_ctx and 0 <= qp < n_ctx:
            col = (i * 5) % dim
            k[key, head // (heads // kv_heads), col] = 5.0
            q[qp, head, col] = 30.0
    k, v, q = k.to(dtype).float(), v.to(dtype).float(), q.to(dtype).float()
    pool = torch.full((2, n_pages + 3, 2, kv_heads, page, dim), float("nan"), dtype=dtype, device=DEV)
    pool[1, perm] = 0.0
    for j in range(n_ctx):
        pool[1, perm[j // page], 0, :, j % page] = k[j].to(dtype)
        pool[1, perm[j // page], 1, :, j % page] = v[j].to(dtype)
    want = P.masked_attention(q.double(), k.double(), v.double(), P.visible(n_ctx, {"size": window, "keep_first": keep}), scale)[positions]
    ctx = _ctx(rt, runs)
    table = torch.full((len(runs), n_pages), -1, dtype=torch.int32)
    for s, (p0, n) in enumerate(runs):
        for pg in range(-(-(p0 + n) // page)):
            if (pg + 1) * page > p0 - window + 1 or pg * page < keep:
                table[s, pg] = int(perm[pg])
    view = KvLayerView(pool, 1, table.to(DEV))
    out = attention.paged_attention(ctx, q[positions].reshape(T, heads * dim).to(DEV, dtype).contiguous(), view, heads, window, scale, keep_first=keep)
    got = out.float().cpu().double().view(T, heads, dim)
    err = (got - want).abs().amax(dim=(1, 2))
    assert err.max().item() < tol, f"positions {[positions[i] for i in torch.nonzero(~(err < tol)).flatten().tolist()]} differ by up to {err.max().item():.2e}"
    rt.check_status()


KEPT = [(4, 2, 64, 16, 48, 5), (16, 1, 128, 16, 100, 20), (2, 2, 128, 64, 64, 64), (6, 3, 64, 8, 130, 1), (4, 4, 64, 32, 1000, 9), (3, 1, 64, 16, 1, 70), (8, 4, 128, 64, 136, 130),
        (4, 2, 32, 16, 24, 4), (5, 5, 24, 8, 13, 40), (8, 1, 64, 64, 65, 300)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,page,window,keep", KEPT)
def test_attention_over_a_window_and_the_first_positions(rt32, rt16, dtype, heads, kv_heads, dim, page, window, keep):
    """bfloat16 heads of 64 and 128 run on the tensor-core kernels (prompt portions and decoded tokens), the rest on the generic one."""
    _kept_case(rt32 if dtype == torch.float32 else rt16, dtype, heads, kv_heads, dim, page, window, keep, 3e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("options", [dict(decode_attention="split"), dict(decode_attention="split", split_tiles_per_slice=1), dict(stream_tiles_per_slice=1), dict(stream_tiles_per_slice=3)])
@pytest.mark.parametrize("heads,kv_heads,dim,page,window,keep", KEPT[:3] + KEPT[6:7])
def test_kept_first_positions_in_every_decode_kernel(options, heads, kv_heads, dim, page, window, keep):
    from inference_bench_b200.config.runtime_options import RuntimeOptions
    from inference_bench_b200.engine.runtime import Runtime
    _kept_case(Runtime(DEV, options=RuntimeOptions(**options)), torch.bfloat16, heads, kv_heads, dim, page, window, keep, 3e-2)


# ------------------------------------------------------------------------------------------ queries and keys of two maps, and their combination
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("interleaved", [True, False])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims,page", [(4, 2, 16, 24, 8, 16), (3, 3, 10, 14, 0, 8), (8, 1, 64, 128, 64, 64), (2, 2, 5, 3, 4, 16), (6, 2, 32, 64, 2, 16)])
def test_rows_of_two_maps(rt32, rt16, dtype, interleaved, heads, kv_heads, dim, vdim, dims, page):
    """Partial sums, biases, the rotation of every map at far positions, queries as zero-padded rows, keys and values in the paged cache, with and
    without keys and values of its own."""
    from inference_bench_b200.kernels import ops
    from inference_bench_b200.kernels.ops import KvLayerView
    rt = rt32 if dtype == torch.float32 else rt16
    g = torch.Generator().manual_seed(heads + dim)
    runs, base = [(0, 5), (3 * page - 2, 4), (700, 1)], 5000.0
    ctx = _ctx(rt, runs)
    T, row = ctx.n_tokens, max(2 * dim, vdim) + max(2 * dim, vdim) % 2
    pos = torch.tensor([p0 + i for p0, n in runs for i in range(n)])
    n_pages = 705 // page + 1
    perm = torch.randperm(n_pages, generator=g)
    table = perm.to(torch.int32).reshape(1, -1).repeat(len(runs), 1).contiguous().to(DEV)
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    cos = sin = None
    if half:
        a = pos.double()[:, None] * f
        cos, sin = _f32(torch.cos(a)), _f32(torch.sin(a))
    for own in (True, False):
        R = heads * 2 * dim + (kv_heads * (2 * dim + vdim) if own else 0)
        parts, bias = torch.randn((3, T, R), generator=g), torch.randn((R,), generator=g)
        z = parts.double().sum(0) + bias.double()
        pool = torch.full((1, n_pages, 2, kv_heads, page, row), 7.0, dtype=dtype, device=DEV)
        q = torch.full((T, heads * 4 * dim), 9.0, dtype=dtype, device=DEV)
        ops.map_qkv(_f32(parts), _f32(bias), cos, sin, interleaved, ctx.positions, ctx.seg_of_token, q, KvLayerView(pool, 0, table), heads, 2, dim, vdim, rt.status, write_kv=own)
        tol = dict(atol=1e-5) if dtype == torch.float32 else dict(rtol=2.0 ** -8, atol=1e-6)
        want = P.rotate(z[:, :heads * 2 * dim].reshape(T, heads * 2, dim), pos, dims, base, interleaved).view(T, heads, 2, dim)
        got = q.cpu().double().view(T, heads, 2, 2, dim)
        assert torch.allclose(got[:, :, 0, 0], want[:, :, 0], **tol) and torch.allclose(got[:, :, 1, 1], want[:, :, 1], **tol)
        assert (got[:, :, 0, 1] == 0).all() and (got[:, :, 1, 0] == 0).all()
        if not own:
            assert (pool == 7.0).all()
            continue
        k = P.rotate(z[:, heads * 2 * dim:(heads + kv_heads) * 2 * dim].reshape(T, kv_heads * 2, dim), pos, dims, base, interleaved).view(T, kv_heads, 2 * dim)
        v = z[:, (heads + kv_heads) * 2 * dim:].view(T, kv_heads, vdim)
        kept = pool.cpu().double()
        for t, p in enumerate(pos.tolist()):
            at = kept[0, perm[p // page], :, :, p % page]
            assert torch.allclose(at[0, :, :2 * dim], k[t], **tol) and torch.allclose(at[1, :, :vdim], v[t], **tol)
    rt.check_status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,heads,vdim", [(1, 2, 24), (19, 3, 14), (300, 8, 128), (7, 1, 3)])
def test_the_difference_of_two_maps(rt32, dtype, T, heads, vdim):
    from inference_bench_b200.kernels import ops
    a = torch.randn((T, heads, 2, vdim), generator=torch.Generator().manual_seed(T)).to(dtype)
    out = torch.empty((T, heads * vdim), dtype=dtype, device=DEV)
    ops.diff_combine(a.reshape(T, -1).to(DEV).contiguous(), 0.37, 1e-5, 0.45, out, vdim)
    want = P.rms_unit(a[:, :, 0].double() - 0.37 * a[:, :, 1].double(), 1e-5) * 0.45
    assert torch.allclose(out.cpu().double().view(T, heads, vdim), want, **(dict(atol=2e-6) if dtype == torch.float32 else dict(rtol=2.0 ** -7, atol=1e-6)))


@pytest.mark.parametrize("heads,kv_heads,dim,page,window,keep", [(4, 2, 64, 16, 48, 5), (16, 1, 128, 16, 100, 20), (6, 3, 128, 64, 1000, 3), (2, 1, 64, 64, None, 0), (4, 2, 24, 8, 13, 40)])
@pytest.mark.parametrize("portion", [0, 5])
def test_the_difference_of_two_maps_where_the_slices_are_merged(rt16, heads, kv_heads, dim, page, window, keep, portion):
    """Decoded tokens from the first positions to a long context, alone (the merge kernel takes the difference and the norm) and beside a prompt
    portion (a kernel of its own does)."""
    from inference_bench_b200.kernels import attention
    from inference_bench_b200.kernels.ops import KvLayerView
    n_ctx, scale, lam, eps, factor = 700, 0.3, 0.6, 1e-5, 0.45
    g = torch.Generator().manual_seed(heads + dim)
    runs = [(0, 1), (1, 1), (keep + 60, 1), (333, 1), (699, 1)] + ([(20, portion)] if portion else [])
    positions = [p0 + i for p0, n in runs for i in range(n)]
    n_pages = -(-n_ctx // page)
    perm = torch.randperm(n_pages, generator=g)
    k, v, q = (torch.randn((n_ctx, h, dim), generator=g).to(torch.bfloat16).double() for h in (kv_heads, kv_heads, heads))
    pool = torch.zeros((1, n_pages, 2, kv_heads, page, dim), dtype=torch.bfloat16, device=DEV)
    for j in range(n_ctx):
        pool[0, perm[j // page], 0, :, j % page] = k[j].to(torch.bfloat16)
        pool[0, perm[j // page], 1, :, j % page] = v[j].to(torch.bfloat16)
    a = P.masked_attention(q, k, v, P.visible(n_ctx, None if window is None else {"size": window, "keep_first": keep}), scale)[positions].view(len(positions), heads // 2, 2, dim)
    want = P.rms_unit(a[:, :, 0] - lam * a[:, :, 1], eps) * factor
    ctx = _ctx(rt16, runs)
    view = KvLayerView(pool, 0, perm.to(torch.int32).reshape(1, -1).repeat(len(runs), 1).contiguous().to(DEV))
    out = attention.paged_attention(ctx, q[positions].reshape(len(positions), heads * dim).to(DEV, torch.bfloat16).contiguous(), view, heads, window, scale, keep_first=keep,
                                    diff=(lam, eps, factor))
    err = (out.cpu().double().view(want.shape) - want).abs().amax(dim=(1, 2))
    assert err.max().item() < 4e-2, f"positions {[positions[i] for i in torch.nonzero(err >= 4e-2).flatten().tolist()]}: {err.max().item():.2e}"
    rt16.check_status()


@pytest.mark.parametrize("parts,T,N,K", [(4, 1, 192, 192), (4, 8, 1024, 1024), (3, 17, 60, 72), (2, 128, 130, 520), (4, 64, 2048, 2048)])
def test_several_products_in_one_launch(rt16, parts, T, N, K):
    from inference_bench_b200.kernels import gemm_tcgen05 as G
    g = torch.Generator().manual_seed(T + N)
    x, w = (torch.randn(s, generator=g).to(torch.bfloat16) for s in ((parts, T, K), (parts, N, K)))
    out = G.gemm_parts(rt16, x.to(DEV), w.to(DEV)).sum(0).cpu().double()
    want = torch.einsum("ptk,pnk->ptn", x.double(), w.double())
    assert (out - want).abs().max().item() < 1e-4 * want.abs().max().item()
    rt16.check_status()


@pytest.mark.parametrize("T,E,groups,keep,top,score,always", [(1, 1, 1, 1, 1, "chosen_softmax", 1), (8, 64, 1, 1, 6, "chosen_softmax", 2), (32, 16, 4, 2, 3, "sigmoid", 0), (5, 40, 1, 1, 40, "softmax", 3),
                                                              (31, 6, 1, 1, 2, "chosen_softmax", 0)])
def test_choice_and_regrouping_in_one_kernel(rt32, T, E, groups, keep, top, score, always):
    """The same choices and weights as the router's own kernel, and rows that lie in their expert's range, each pair in one of its own."""
    from inference_bench_b200.kernels import ops
    g = torch.Generator().manual_seed(T + E)
    logits, bias = _f32(torch.randn((2, T, E + 1), generator=g)), _f32(torch.randn((E,), generator=g))
    R, n = T * (top + always), E + always
    new = lambda *shape: torch.empty(shape, dtype=torch.int32, device=DEV)
    got = []
    for fused in (False, True):
        idx, wt, off, tiles, row, tok = new(T, top + always), torch.empty((T, top + always), device=DEV), new(n + 1), new(n + 1), new(R), new(R)
        ops.moe_route(logits, groups, keep, top, 1.5, score == "softmax", idx, wt, score, experts=E, logit_bias=bias, always=always, gate_col=E if always else -1,
                      sort=(off, tiles, row, tok, 16) if fused else None)
        if not fused:
            ops.moe_sort(idx, n, off, tiles, row, tok, tile_rows=16)
        got.append([t.cpu() for t in (idx, wt, off, tiles)])
        idx, off, row, tok = idx.cpu().flatten(), off.cpu(), row.cpu(), tok.cpu()
        assert sorted(row.tolist()) == list(range(R)) and int(off[-1]) == R
        for pair in range(R):
            e = int(idx[pair])
            assert off[e] <= row[pair] < off[e + 1] and int(tok[row[pair]]) == pair // (top + always)
    for a, b in zip(*got):
        assert torch.equal(a, b)
    z = logits.cpu().double().sum(0)
    if always:
        assert torch.allclose(got[0][1][:, top:].double(), torch.sigmoid(z[:, E:]).expand(T, always), atol=1e-6)
    if score == "chosen_softmax":
        best = torch.topk(z[:, :E] + bias.cpu().double(), top).values
        assert torch.allclose(got[0][1][:, :top].double(), 1.5 * torch.softmax(best, -1), atol=1e-5)
    rt32.check_status()


# ------------------------------------------------------------------------------------------ recurrences over portions and slots
def _walk_part(rt, plan, part, mixer, want_fn, W, caches, zero, run, tol):
    g = torch.Generator().manual_seed(W)
    lens = _lens(plan)
    x = {r: torch.randn((n, W), generator=g).to(torch.bfloat16) for r, n in lens.items()}
    want = {r: want_fn(x[r].double()) for r in lens}
    with P.rounded():
        moved = {r: (want_fn(x[r].double()) - want[r]).abs().amax(dim=1) / want[r].abs().max() for r in lens}

    def step_fn(ctx, step, at):
        xs = torch.cat([x[r][at[r]:at[r] + n] for r, n in step]).to(DEV)
        out = run(ctx, xs).sum(0).cpu().double()
        o = 0
        for r, n in step:
            err = (out[o:o + n] - want[r][at[r]:at[r] + n]).abs().amax(dim=1) / want[r].abs().max().item()
            if rt.mode == "bfloat16":    # what rounding alone moves a row by in the plain form, times four, where that is more
                err = err * torch.clamp(tol / (4.0 * moved[r][at[r]:at[r] + n]), max=1.0)
            assert err.max().item() < tol, f"request {r} rows {at[r]}..{at[r] + n}: row {at[r] + int(err.argmax())} differs by {err.max().item():.2e}"
            o += n

    _steps(rt, plan, SLOTS, ("c",), zero, step_fn)
    rt.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("long_segments", [False, True])
@pytest.mark.parametrize("heads,dim,vdim,dims,decay", [(3, 20, 12, 12, (0.5, 0.9, 0.99)), (4, 12, 40, 12, (1.0, 0.0, 0.8, 0.999)), (2, 64, 128, 32, (0.98, 0.6)), (2, 34, 6, 0, (0.97, 0.3)),
                                                       (1, 300, 20, 2, (0.95,))])
def test_retention_over_portions_and_slots(dtype, long_segments, heads, dim, vdim, dims, decay):
    """The mixer as a part, its state slots by hand: portions of 1, 2 and more tokens of three requests in two slots, or portions just below, at
    and above multiples of a chunk, from zero and from earlier states, equal the plain recurrence over each whole sequence."""
    from inference_bench_b200.cache.manager import StateView
    from inference_bench_b200.engine.runtime import Runtime
    from inference_bench_b200.kernels.ops import RECURRENCE_CHUNK
    from inference_bench_b200.parts.retention import Retention
    from inference_bench_b200.parts.standard import NoPositionEncoding, RotaryEmbedding
    rt, W = Runtime(DEV, dtype=dtype), 64
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": {"base": 300.0, "dims": dims}}
    w = tf.tensors({"vocab": 8, "width": W, "layers": [{"type": "retention", "mixer": m, "mlp": None}]}, dim)
    part = Retention("l0.mix", W, heads, dim, vdim, decay, 1e-5, RotaryEmbedding(dims, 300.0) if dims else NoPositionEncoding())
    part.bind({n: t.to(DEV) for n, t in w.items()}, rt)
    state = torch.zeros((3, heads, dim, vdim), device=DEV)
    _walk_part(rt, _long(RECURRENCE_CHUNK) if long_segments else SHORT, part, m, lambda x: P.retention(x, w, "l0.mix", m, 1e-5), W, None, lambda s: state[s].zero_(),
               lambda ctx, xs: part.forward(ctx, xs.to(rt.act_dtype).contiguous(), StateView(state)), 5e-5 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("long_segments", [False, True])
@pytest.mark.parametrize("W,heads,dim,rank", [(80, 3, 20, 3), (132, 5, 24, 1), (192, 3, 64, 24), (64, 1, 130, 70), (48, 2, 270, 5)])
def test_wkv_over_portions_and_slots(dtype, long_segments, W, heads, dim, rank):
    """The same for the recurrence behind a token shift: the mixer runs its norm, the residual add (a scaled contribution) and the five mixes; a
    lost previous row, a decay that reaches the current token's own output or a bonus that stays in the state would show."""
    from inference_bench_b200.cache.manager import StateView
    from inference_bench_b200.engine.runtime import Runtime
    from inference_bench_b200.kernels.ops import RECURRENCE_CHUNK
    from inference_bench_b200.parts.base import ScaledDelta
    from inference_bench_b200.parts.retention import WkvMixer
    from inference_bench_b200.parts.standard import LayerNorm
    rt = Runtime(DEV, dtype=dtype)
    m = {"heads": heads, "dim": dim}
    w = tf.tensors({"vocab": 8, "width": W, "layers": [{"type": "wkv", "mixer": m, "mlp": None}]}, dim, rank)
    dev = {n: t.to(DEV) for n, t in w.items()}
    norm, part = LayerNorm("l0.norm1", W, 1e-5, bias="{}.b"), WkvMixer("l0.mix", W, heads, dim, 1e-5)
    norm.bind(dev, rt), part.bind(dev, rt)
    state, last = torch.zeros((3, heads, dim, dim), device=DEV), torch.zeros((3, W), device=DEV)

    def run(ctx, xs):
        xd = _f32(xs)
        delta = torch.stack([xd * 0.5, xd * 0.25]).contiguous()
        x = (xd - 0.4 * delta.sum(0)).contiguous()          # the stream before the contribution is added
        out = part.forward_normed(ctx, norm, x, ScaledDelta(delta, 0.4), (StateView(state), StateView(last)))
        assert torch.allclose(x, xd, atol=1e-5)
        return out

    def zero(s):
        state[s].zero_(), last[s].zero_()

    want = lambda x: P.wkv(P.layer_norm(x, w, "l0.norm1", 1e-5), w, "l0.mix", m, 1e-5)
    _walk_part(rt, _long(RECURRENCE_CHUNK) if long_segments else SHORT, part, m, want, W, None, zero, run, 5e-5 if dtype == "float32" else 5e-2)


# ------------------------------------------------------------------------------------------ norms, embedding, cap, experts
@pytest.mark.parametrize("H", [48, 132, 1022, 4096])
def test_layer_norm_with_bias_scaled_contribution_and_gathered_rows(rt32, rt16, H):
    from inference_bench_b200.parts.base import ScaledDelta
    from inference_bench_b200.parts.standard import LayerNorm, TokenEmbedding
    g = torch.Generator().manual_seed(H)
    T, V = 21, 40
    w = {"n": 1 + 0.2 * torch.randn((H,), generator=g), "n.b": torch.randn((H,), generator=g), "e": torch.randn((V, H), generator=g).to(torch.bfloat16)}
    x, delta = torch.randn((T, H), generator=g) * 3 + 1, torch.randn((3, T, H), generator=g)
    summed = x.double() + 0.37 * delta.double().sum(0)
    rows = [20, 3, 3, 0]
    for rt, tol in ((rt32, dict(atol=3e-5)), (rt16, dict(rtol=2.0 ** -8, atol=1e-3))):
        norm = LayerNorm("n", H, 1e-5, bias="{}.b")
        norm.bind({n: t.to(DEV) for n, t in w.items()}, rt)
        for ctx in (_ctx(rt, [(0, T)]), _ctx(rt, [(i, 1) for i in range(T)])):
            xd = _f32(x)
            out = norm.forward(ctx, xd, ScaledDelta(_f32(delta), 0.37))
            assert torch.allclose(out.cpu().double(), P.layer_norm(summed, w, "n", 1e-5), **tol) and torch.allclose(xd.cpu().double(), summed, atol=1e-5)
            xd = _f32(x)
            out = norm.forward(ctx, xd, ScaledDelta(_f32(delta), 0.37), rows=torch.tensor(rows, dtype=torch.int32, device=DEV))
            assert torch.allclose(out.cpu().double(), P.layer_norm(summed, w, "n", 1e-5)[rows], **tol) and torch.equal(xd.cpu(), x)
        emb = TokenEmbedding("e", V, H, norm=LayerNorm("n", H, 1e-5, bias="{}.b"))
        emb.bind({n: t.to(DEV) for n, t in w.items()}, rt)
        ctx = _ctx(rt, [(0, 4)])
        ctx.token_ids.copy_(torch.tensor([7, 0, 39, 7], dtype=torch.int32))
        got = emb.forward(ctx)
        assert got.dtype == torch.float32 and torch.allclose(got.cpu().double(), P.layer_norm(w["e"].double()[[7, 0, 39, 7]], w, "n", 1e-5), atol=3e-5)
        rt.check_status()


def test_capped_values(rt32):
    from inference_bench_b200.kernels import ops
    v = torch.tensor([0.0, -3.0, 1e-3, 50.0, -500.0, 29.0])
    got = _f32(v)
    ops.softcap_values(got, 30.0)
    assert torch.allclose(got.cpu().double(), 30.0 * torch.tanh(v.double() / 30.0), atol=1e-5)


@pytest.mark.parametrize("T,N,K", [(1, 4096, 64), (8, 4224, 1024), (5, 200, 72), (64, 5000, 520), (128, 130, 64), (8, 256, 2048), (129, 520, 264), (700, 8192, 256), (2048, 384, 512),
                                   (2300, 1100, 72)])
def test_product_with_squared_relu(rt16, T, N, K):
    """The activation on the float32 accumulators in the tensor-core kernels' epilogues (or in the row-wise kernel where the k-range is cut),
    against float64."""
    g = torch.Generator().manual_seed(T + N + K)
    x = (torch.randn(T, K, generator=g) * 0.7).to(torch.bfloat16).to(DEV)
    lw = rt16.matrix((torch.randn(N, K, generator=g) * (2.0 / math.sqrt(K))).to(torch.bfloat16))
    act = rt16.up_act(x, lw, "relu2")
    want = P.relu2(x.cpu().double() @ lw.weight.cpu().double().T)
    assert ((act.cpu().double() - want).abs() <= 2.0 ** -8 * want.abs() + 2e-5 * want.abs().max()).all()
    rt16.check_status()


@pytest.mark.parametrize("dtype,how", [("float32", "auto"), ("bfloat16", "auto"), ("bfloat16", "mma"), ("bfloat16", "simt")])
@pytest.mark.parametrize("W,ff,experts,top,shared", [(80, 24, 5, 2, 56), (132, 36, 1, 1, 20), (132, 28, 3, 1, None), (192, 64, 16, 4, 128), (192, 128, 6, 6, 64), (64, 40, 40, 3, 8)])
def test_experts_with_squared_relu(dtype, how, W, ff, experts, top, shared):
    """Routing by biased logits, softmax over the chosen ones, experts without a gate, the shared expert's gate; one token to several hundred.
    Rows whose choice of the last expert is close are left out in bfloat16."""
    from inference_bench_b200.config.runtime_options import RuntimeOptions
    from inference_bench_b200.engine.runtime import Runtime
    from inference_bench_b200.parts.experts import RoutedExperts
    rt = Runtime(DEV, options=RuntimeOptions(dtype=dtype, expert_gemm=how))
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": None if shared is None else {"ff": shared}}
    cfg = {"vocab": 8, "width": W, "layers": [{"type": "wkv", "mixer": {"heads": 1, "dim": 4}, "mlp": f}]}
    w = tf.tensors(cfg, ff + experts)
    part = RoutedExperts("l0.mlp", W, ff, experts, top, shared_ff=shared or 0, score="chosen_softmax", activation="relu2", router_bias="router.b", shared_gate="sg")
    assert {s.name for s in part.weight_specs()} == {n for n in w if n.startswith("l0.mlp")}
    part.bind({n: t.to(DEV) for n, t in w.items()}, rt)
    g = torch.Generator().manual_seed(W)
    for T in (1, 3, 37, 300):
        h = torch.randn((T, W), generator=g).to(torch.bfloat16)
        out = part.forward(_ctx(rt, [(0, T)]), h.to(DEV, rt.act_dtype).contiguous()).sum(0).cpu().double()
        want = P.experts_ff(h.double(), w, "l0.mlp", f)
        err = (out - want).abs().amax(1) / want.abs().max()
        if dtype == "bfloat16" and top < experts:
            z = torch.sort(h.double() @ w["l0.mlp.router"].double().T + w["l0.mlp.router.b"].double(), descending=True).values
            err = err[(z[:, top - 1] - z[:, top]) > 1e-2]
        assert err.numel() == 0 or err.max().item() < (2e-5 if dtype == "float32" else 2e-2), f"{T} tokens: {err.max().item():.2e}"
    rt.check_status()


# ------------------------------------------------------------------------------------------ whole models
def _requests(name):
    vocab = tf.CONFIGS[name]["config"]["vocab"]
    return {r: traces.prompt(500 + i, n, vocab) for i, (r, n) in enumerate({"a": 150, "b": 1, "c": 23, "d": 64, "e": 97, "f": 2}.items())}


@pytest.fixture(scope="module")
def plain_logits(fdirs):
    return {name: {r: P.PlainFedipel(fdirs[name]).logits(t).numpy() for r, t in _requests(name).items()} for name in tf.CONFIGS}


@pytest.fixture(scope="module")
def rounded_logits(fdirs):
    with P.rounded():
        return {name: {r: P.PlainFedipel(fdirs[name]).logits(t).numpy() for r, t in _requests(name).items()} for name in tf.CONFIGS}


def _runner(model_dir, dtype, max_tokens, page_size, **kw):
    from inference_bench_b200.trace import build_runner
    return build_runner(model_dir, dtype, max_tokens, page_size=page_size, **kw)


def _compare(got, want_by_req, dtype, what, moved=None):
    """float32: every row. bfloat16: a row may differ by as much as TOLERANCE, or by four times what rounding alone moves it in the plain model
    (`moved`: a head's norm after a difference of two nearly equal maps, or of a first token's small output, enlarges it), except for one row in
    fifty (a router's close call), and half the rows are far closer."""
    errs, over = [], []
    for (r, pos), row in got.items():
        span = np.abs(want_by_req[r]).max()
        err = np.abs(row - want_by_req[r][pos]).max() / span
        errs.append(err)
        if not err <= max(TOLERANCE[dtype], 0.0 if moved is None else 4.0 * np.abs(moved[r][pos] - want_by_req[r][pos]).max() / span):
            over.append((r, pos, float(err)))
    assert len(got) == sum(len(v) for v in want_by_req.values())
    assert len(over) <= (0 if dtype == "float32" else 0.02 * len(got)), f"{what}: rows over their limit: {over}"
    if dtype == "bfloat16":
        assert float(np.median(errs)) < BF16_MEDIAN, f"{what}: the median row differs by {np.median(errs):.2e} of max|logit|"
    return max(errs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tf.CONFIGS))
def test_layers_one_by_one(fdirs, name, dtype):
    """The residual stream after every layer against the plain model's, so that a wrong layer is named."""
    from inference_bench_b200.engine.step import StepEntry
    toks = _requests(name)["e"]
    want = P.PlainFedipel(fdirs[name]).hidden_states(toks)
    runner = _runner(fdirs[name], dtype, 128, tf.CONFIGS[name]["page_size"])
    runner.cache.admit("x")
    layers = []
    runner.step([StepEntry("x", toks, list(range(len(toks))))], trace=layers)
    assert len(layers) == len(want) + 1
    for i, (g, w) in enumerate(zip(layers[1:], want)):
        err = (g.cpu().double() - w).abs().amax(dim=1) / w.abs().max().item()
        if dtype == "bfloat16":     # a router's close call may fall the other way in a few rows, a head's norm may enlarge rounding
            err = err.sort().values[:int(0.9 * len(toks))]
        assert err.max().item() < (2e-5 if dtype == "float32" else 4e-2), f"{name}/{dtype}: the stream after layer {i} differs by {err.max().item():.2e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tf.CONFIGS))
@pytest.mark.parametrize("cut", ["whole", "tail", "portions", "mixed"])
def test_cut_matches_plain(fdirs, plain_logits, rounded_logits, name, dtype, cut):
    """Whole prompts; prompts then the last tokens one by one (a tail long enough for every window to pass over decoded tokens only); portions
    down to two tokens; up to four live requests of unequal length in one batch with a pool that only holds what is live, so pages and slots
    are used again by later requests."""
    reqs = _requests(name)
    steps = {"whole": traces.whole, "tail": lambda r: traces.tail_one_by_one(r, tail=80), "portions": traces.portions, "mixed": traces.mixed}[cut](reqs)
    max_tokens = traces.max_live_tokens(steps)
    runner = _runner(fdirs[name], dtype, max_tokens, tf.CONFIGS[name]["page_size"], max_requests=4)
    got = traces.run_steps(runner, steps)
    worst = _compare(got, plain_logits[name], dtype, f"{name}/{dtype}/{cut}", rounded_logits[name] if dtype == "bfloat16" else None)
    runner.cache.check()
    assert runner.cache.used_pages() == [0] * len(runner.cache.groups)
    print(f"{name}/{dtype}/{cut}: worst {worst:.3e} of max|logit|, pool {max_tokens} tokens")


@pytest.mark.parametrize("name", ["A", "C"])
def test_a_request_alone_and_in_a_batch_give_the_same_float32_logits(fdirs, name):
    """The float32 path adds in one order whatever shares the step: a request beside three others of other lengths, on other pages and
    in another slot, gives the bits it gives alone."""
    from inference_bench_b200.engine.step import StepEntry
    reqs = _requests(name)
    runner = _runner(fdirs[name], "float32", 1024, 16, max_requests=4)
    runner.cache.admit("alone")
    alone = runner.step([StepEntry("alone", reqs["d"], [len(reqs["d"]) - 1])]).cpu()
    runner.cache.release("alone")
    for r in ("c", "f", "d", "a"):
        runner.cache.admit(r)
    rows = runner.step([StepEntry(r, reqs[r], [len(reqs[r]) - 1]) for r in ("c", "f", "d", "a")]).cpu()
    assert torch.equal(rows[2], alone[0])


# ------------------------------------------------------------------------------------------ weights made so that a fault shows
def _one_layer(tmp_path, mask, gain, tag, second=None):
    """One attention layer (and optionally a reader of its keys) without a feed-forward; queries and keys scaled so that each softmax nearly picks
    one key."""
    att = {"heads": 2, "kv_heads": 1, "dim": 16, "vdim": 32, "mask": mask, "rot": {"base": 100.0, "dims": 8}, "scale": gain, "diff": 0.4}
    layers = [{"type": "attention", "mixer": att, "mlp": None}]
    if second is not None:
        layers.append({"type": "attention", "mixer": dict(att, mask=second, kv_from=0), "mlp": None})
    cfg = {"architecture": "Fedipel", "vocab": 64, "width": 40, "norm": {"eps": 1e-6}, "residual_mult": 1.0, "logit_softcap": None, "layers": layers}
    return tf.write_folder(tmp_path / tag, cfg, tf.tensors(cfg, 77))


@pytest.mark.parametrize("size,keep,second,page", [(16, 3, None, 16), (7, 20, None, 16), (33, 1, (50, 9), 8), (20, 4, (6, 4), 16), (1, 2, None, 8)])
def test_keys_just_inside_and_just_outside_what_is_seen(tmp_path, size, keep, second, page):
    """With softmaxes that nearly pick one key, a window or a run of kept positions that is one off changes many rows by far more than the tolerance;
    the engine equals the right mask for whole prompts and for tokens decoded one by one, also where a second layer reads the same keys with a
    mask of its own."""
    from inference_bench_b200.engine.step import StepEntry
    mask = {"size": size, "keep_first": keep}
    model = _one_layer(tmp_path, mask, 8.0, "m", None if second is None else {"size": second[0], "keep_first": second[1]})
    plain = P.PlainFedipel(model)
    toks = traces.prompt(11, 130, 64)
    want = plain.logits(toks)
    n = len(plain.cfg["layers"])
    for layer, key, off in [(i, k, o) for i in range(n) for k, o in (("size", 1), ("size", -1), ("keep_first", 1), ("keep_first", -1))]:
        bad = copy.deepcopy(plain.cfg)
        m = bad["layers"][layer]["mixer"]["mask"]
        m[key] += off
        if m["size"] < 1:
            continue
        diff = (P.logits(bad, plain.w, toks) - want).abs().amax(dim=1) / want.abs().max()
        assert int((diff > 0.02).sum()) >= 2, f"{key} {off:+d} in layer {layer} would not show ({diff.max().item():.2e})"
    for head in (len(toks), size + keep + 2, 1):
        runner = _runner(model, "float32", 256, page)
        runner.cache.admit("x")
        rows = [runner.step([StepEntry("x", toks[:head], list(range(head)))]).cpu()]
        rows += [runner.step([StepEntry("x", [t], [0])]).cpu() for t in toks[head:]]
        err = (torch.cat(rows).double() - want).abs().amax(dim=1) / want.abs().max()
        assert err.max().item() < 2e-4, f"prompt of {head} then one by one: {err.max().item():.2e} at position {int(err.argmax())}"


def test_the_first_token_counts_for_ever(tmp_path):
    """A head whose decay is 1 and a kept first position: the first token still moves the logits 400 tokens on, through the chunked form, the
    attention over kept pages and single tokens alike."""
    from inference_bench_b200.engine.step import StepEntry
    att = {"heads": 2, "kv_heads": 2, "dim": 8, "vdim": 16, "mask": {"size": 5, "keep_first": 1}, "rot": {"base": 100.0, "dims": 4}, "scale": 0.2, "diff": 0.4}
    ret = {"heads": 2, "dim": 8, "vdim": 8, "decay": [1.0, 0.97], "rot": {"base": 1e6, "dims": 4}}
    for tag, kind, mixer in (("att", "attention", att), ("ret", "retention", ret)):
        cfg = {"architecture": "Fedipel", "vocab": 64, "width": 40, "norm": {"eps": 1e-6}, "residual_mult": 1.0, "logit_softcap": 30.0,
               "layers": [{"type": kind, "mixer": mixer, "mlp": None}]}
        model = tf.write_folder(tmp_path / tag, cfg, tf.tensors(cfg, 78))
        plain = P.PlainFedipel(model)
        toks = traces.prompt(12, 400, 64)
        want = plain.logits(toks)
        other = list(toks)
        other[0] = (toks[0] + 1) % 64
        assert ((plain.logits(other) - want)[-8:].abs().amax(dim=1) / want.abs().max()).median().item() > 1e-3
        for head in (400, 330):
            runner = _runner(model, "float32", 448, 16)
            runner.cache.admit("x")
            rows = [runner.step([StepEntry("x", toks[:head], list(range(head)))]).cpu()]
            rows += [runner.step([StepEntry("x", [t], [0])]).cpu() for t in toks[head:]]
            err = (torch.cat(rows).double() - want).abs().amax(dim=1) / want.abs().max()
            assert err.max().item() < 1e-4, f"{tag} {head}: {err.max().item():.2e} at {int(err.argmax())}"


# ------------------------------------------------------------------------------------------ generation
@pytest.mark.parametrize("name", list(tf.CONFIGS))
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_engine(fdirs, name, graphs):
    """`Engine.generate`: the scheduler cuts prompts into portions, batches them beside decoded tokens, and decode steps run as captured
    graphs or not; float32 tokens equal the plain model's."""
    from inference_bench_b200 import Engine
    vocab = tf.CONFIGS[name]["config"]["vocab"]
    plain = P.PlainFedipel(fdirs[name])
    prompts = [traces.prompt(90 + i, n, vocab) for i, n in enumerate((5, 21, 40))]
    want = [plain.greedy(p, 7) for p in prompts]
    eng = Engine(fdirs[name], dtype="float32", max_ctx=128, page_size=tf.CONFIGS[name]["page_size"], use_graphs=graphs, prefill_chunk=9, max_batched_tokens=16)
    got = eng.generate(prompts, max_tokens=7)
    assert [r.tokens for r in got] == want
    assert eng.cache.used_pages() == [0] * len(eng.cache.groups)
    eng.cache.check()
    one = eng.generate(prompts[1], max_tokens=7)
    assert one.tokens == want[1]


def test_generation_in_bfloat16_runs_and_long_decoding_stays_close(fdirs):
    from inference_bench_b200 import Engine
    name = "C"
    vocab = tf.CONFIGS[name]["config"]["vocab"]
    plain = P.PlainFedipel(fdirs[name])
    prompt = traces.prompt(5, 12, vocab)
    eng = Engine(fdirs[name], dtype="bfloat16", max_ctx=256, page_size=16)
    got = eng.generate(prompt, max_tokens=120).tokens
    assert len(got) == 120
    lg = plain.logits(prompt + got)     # teacher-forced on the engine's own tokens, the plain model ranks every chosen token near the top
    span = float(lg.max() - lg.min())
    below = [float(lg[len(prompt) + i - 1].max() - lg[len(prompt) + i - 1][tok]) / span for i, tok in enumerate(got)]
    assert all(math.isfinite(b) for b in below) and max(below) < 0.2
    assert sum(b > 0.03 for b in below) <= 0.1 * len(got)


def test_trace_replay_program_and_command_line(fdirs, tmp_path):
    """bin/trace_run as a subprocess fed JSON steps (a mixed trace, float32), and `run` and `spec` of the command line, on a model folder
    of this architecture: nothing in them names an architecture."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    name = "A"
    vocab = tf.CONFIGS[name]["config"]["vocab"]
    reqs = {r: traces.prompt(900 + i, n, vocab) for i, (r, n) in enumerate({"a": 70, "b": 9, "c": 33, "d": 64, "e": 2}.items())}
    steps = traces.mixed(reqs, seed=5)
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(fdirs[name]), "--dtype", "float32", "--out", str(out),
                           "--max-tokens", str(traces.max_live_tokens(steps))],
                          input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    plain = P.PlainFedipel(fdirs[name])
    want = {r: plain.logits(t).numpy() for r, t in reqs.items()}
    at = {r: 0 for r in reqs}
    for s in steps:
        rows = np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, vocab)
        k = 0
        for e in s["entries"]:
            for w in e["want"]:
                err = np.abs(rows[k] - want[e["id"]][at[e["id"]] + w]).max() / np.abs(want[e["id"]]).max()
                assert err <= TOLERANCE["float32"]
                k += 1
            at[e["id"]] += len(e["tokens"])
        assert k == rows.shape[0]
    env = dict(os.environ, PYTHONPATH=root)
    p = subprocess.run([sys.executable, "-m", "inference_bench_b200", "run", "--model", str(fdirs[name]), "--prompt-len", "12", "--max-tokens", "5", "--json",
                        "--dtype", "float32", "--max-ctx", "64"], capture_output=True, text=True, env=env, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    r = json.loads(p.stdout)
    from inference_bench_b200.cli import _synthetic_prompt
    assert r["prompt_tokens"] == 12 and r["tokens"] == plain.greedy(_synthetic_prompt(12, vocab), 5)
    p = subprocess.run([sys.executable, "-m", "inference_bench_b200", "spec", "--model", str(fdirs[name])], capture_output=True, text=True, env=env)
    assert p.returncode == 0 and json.loads(p.stdout)["layers"][2]["mixer"]["mask"] == {"size": 40, "keep_first": 1}
