"""Gokosun in the engine against the plain implementation: each mechanism's kernels alone (with weights or inputs made so that a far key, a lost
sink, a lost state or a wrong maximum shows), then whole models under every way of cutting the work (in true 32-bit and in bfloat16), pages and
slots that are used again, and greedy generation through the engine's entry point and scheduler."""
from __future__ import annotations

import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_gokosun as P
import tiny_gokosun as tg
import traces

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
F64 = torch.float64
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
def gdirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("gokosun")
    return {name: tg.write_model(name, root / name) for name in tg.CONFIGS}


def _f32(t):
    return t.to(DEV, torch.float32).contiguous()


def _ctx(rt, runs, slots=None):
    """A step's context for segments given as (first position, tokens)."""
    from inference_bench_b200.engine.context import Segment, build_context
    return build_context(rt, [Segment(i, (slots[i] if slots else i), p0, [0] * n, []) for i, (p0, n) in enumerate(runs)])


def _layer_tensors(kind, mixer, W, seed):
    return tg.tensors({"vocab": 8, "width": W, "layers": [{"type": kind, "mixer": mixer, "mlp": None}]}, seed)


# ------------------------------------------------------------------------------------------ the block, its norm, the rotation's tables
@pytest.mark.parametrize("H", [48, 132, 1022, 4096])
def test_layer_norm_adds_two_contributions(rt32, rt16, H):
    from inference_bench_b200.parts.base import SummedDelta
    from inference_bench_b200.parts.standard import LayerNorm
    g = torch.Generator().manual_seed(H)
    T = 21
    w = {"n": 1 + 0.2 * torch.randn((H,), generator=g), "n.b": torch.randn((H,), generator=g)}
    x, a, b = torch.randn((T, H), generator=g) * 3 + 1, torch.randn((3, T, H), generator=g), torch.randn((2, T, H), generator=g)
    summed = x.double() + a.double().sum(0) + b.double().sum(0)
    rows = [20, 3, 3, 0]
    for rt, tol in ((rt32, dict(atol=3e-5)), (rt16, dict(rtol=2.0 ** -8, atol=1e-3))):
        norm = LayerNorm("n", H, 1e-5, bias="{}.b")
        norm.bind({n: t.to(DEV) for n, t in w.items()}, rt)
        for ctx in (_ctx(rt, [(0, T)]), _ctx(rt, [(i, 1) for i in range(T)])):
            xd = _f32(x)
            out = norm.forward(ctx, xd, SummedDelta(_f32(a), _f32(b)))
            assert torch.allclose(out.cpu().double(), P.layer_norm(summed, w, "n", 1e-5), **tol) and torch.allclose(xd.cpu().double(), summed, atol=1e-5)
            xd = _f32(x)
            out = norm.forward(ctx, xd, SummedDelta(_f32(a), _f32(b)), rows=torch.tensor(rows, dtype=torch.int32, device=DEV))
            assert torch.allclose(out.cpu().double(), P.layer_norm(summed, w, "n", 1e-5)[rows], **tol) and torch.equal(xd.cpu(), x)


@pytest.mark.parametrize("T,W,ff", [(5, 80, 40), (300, 192, 520), (2300, 256, 264)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_both_sublayers_read_the_same_rows(dtype, T, W, ff):
    """A block of two layers: the second norm adds what both sublayers of the first left, whether a product added it to the stream itself or not."""
    from inference_bench_b200.cache.manager import StateView
    from inference_bench_b200.engine.runtime import Runtime
    from inference_bench_b200.parts.memory import MatrixMemory
    from inference_bench_b200.parts.standard import LayerNorm, NoNorm, ParallelBlock, SwiGLU
    rt = Runtime(DEV, dtype=dtype)
    m = {"heads": 2, "dim": 16, "vdim": 24, "gate_cap": 6.0}
    cfg = {"vocab": 8, "width": W, "norm": {"eps": 1e-5}, "layers": [{"type": "mlstm", "mixer": m, "mlp": {"kind": "dense", "ff": ff, "limit": 1.5}}] * 2}
    w = tg.tensors(cfg, W)
    dev = {n: t.to(DEV) for n, t in w.items()}
    x = torch.randn((T, W), generator=torch.Generator().manual_seed(T)).double()
    xd, pending = _f32(x), None
    ctx = _ctx(rt, [(0, T)])
    run = lambda: P.hidden_from(cfg, w, x)[-1]
    want = run()
    with P.rounded():
        moved = (run() - want).abs().amax(1) / want.abs().max()
    for i in range(2):
        norm = LayerNorm(f"l{i}.norm1", W, 1e-5, bias="{}.b")
        block = ParallelBlock(norm, MatrixMemory(f"l{i}.mix", W, 2, 16, 24, 6.0, 1e-5), NoNorm(), SwiGLU(f"l{i}.mlp", W, ff, ("gate", "up", "down"), clamp=(1.5, 1.702)))
        for p in block.parts():
            p.bind(dev, rt)
        cache = (StateView(torch.zeros((1, 2, 16, 25), device=DEV)), StateView(torch.zeros((1, 2), device=DEV)))
        pending = block.forward(ctx, xd, pending, cache)
    final = LayerNorm("final.norm", W, 1e-5, bias="{}.b")
    final.bind(dev, rt)
    final.forward(ctx, xd, pending)
    err = (xd.cpu().double() - want).abs().amax(1) / want.abs().max()
    if dtype == "bfloat16":    # a head's norm enlarges rounding where its output is small: what rounding alone moves a row by, times four, where that is more
        assert err.median().item() < 1e-2
        err = (err * torch.clamp(3e-2 / (4.0 * moved), max=1.0)).sort().values[:int(0.995 * T)]
    assert err.max().item() < (2e-5 if dtype == "float32" else 3e-2), f"{err.max().item():.2e}"
    rt.check_status()


@pytest.mark.parametrize("dims,base,yarn", [(16, 1000.0, (4.0, 64, 8.0, 1.0)), (64, 10000.0, (8.0, 4096, 32.0, 1.0)), (8, 50.0, (16.0, 32, 2.0, 0.25)), (4, 300.0, (2.0, 1, 64.0, 32.0)),
                                            (6, 2.0, (40.0, 100000, 4.0, 2.0)), (32, 500000.0, (1.0, 512, 32.0, 1.0))])
def test_rescaled_rotation_tables(rt32, dims, base, yarn):
    from inference_bench_b200.parts.standard import RotaryEmbedding
    part = RotaryEmbedding(dims, base, "interleaved", yarn=yarn)
    part.bind({}, rt32)
    ctx = _ctx(rt32, [(0, 4), (1023, 3), (9000, 1)])
    cos, sin = part.tables(ctx)
    f, amp = P.yarn_frequencies(dims, base, dict(zip(("factor", "original", "fast", "slow"), yarn)))
    a = torch.tensor([0, 1, 2, 3, 1023, 1024, 1025, 9000], dtype=F64)[:, None] * f
    assert torch.allclose(cos.cpu().double(), torch.cos(a) * amp, atol=2e-3 * amp) and torch.allclose(sin.cpu().double(), torch.sin(a) * amp, atol=2e-3 * amp)
    assert torch.allclose(cos.cpu().double()[:7], torch.cos(a[:7]) * amp, atol=2e-4 * amp)
    plain = RotaryEmbedding(dims, base, "interleaved")
    plain.bind({}, rt32)
    assert torch.allclose(plain.tables(ctx)[0].cpu().double()[:4], torch.cos(a[:4, :1] * 0 + torch.arange(4)[:, None] * P.yarn_frequencies(dims, base, None)[0]), atol=1e-5)


# ------------------------------------------------------------------------------------------ attention: whole-row norms, mixed values
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("mix", [None, 0.3, 1.0])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims,page", [(4, 2, 16, 24, 8, 16), (3, 3, 10, 14, 0, 8), (8, 1, 64, 64, 64, 64), (2, 2, 5, 3, 4, 16), (6, 2, 128, 48, 32, 16), (16, 4, 128, 128, 128, 16)])
def test_rows_normed_whole_and_values_mixed(rt32, rt16, dtype, mix, heads, kv_heads, dim, vdim, dims, page):
    """Partial sums, the norms over all heads at once, the rotation at far positions, values as they are or mixed, in the paged cache; the values as
    projected kept for later layers."""
    from inference_bench_b200.kernels import ops
    from inference_bench_b200.kernels.ops import KvLayerView
    rt = rt32 if dtype == torch.float32 else rt16
    g = torch.Generator().manual_seed(heads + dim)
    runs, rot, eps = [(0, 5), (3 * page - 2, 4), (700, 1)], {"dims": dims, "base": 5000.0}, 1e-3
    ctx = _ctx(rt, runs)
    T, row = ctx.n_tokens, max(dim, vdim) + max(dim, vdim) % 2
    pos = torch.tensor([p0 + i for p0, n in runs for i in range(n)])
    n_pages = 705 // page + 1
    perm = torch.randperm(n_pages, generator=g)
    table = perm.to(torch.int32).reshape(1, -1).repeat(len(runs), 1).contiguous().to(DEV)
    nq, nk, nv = heads * dim, kv_heads * dim, kv_heads * vdim
    parts = torch.randn((3, T, nq + nk + nv), generator=g) * torch.linspace(0.2, 3.0, nq + nk + nv)     # heads of unequal size: a norm per head would show
    z, qw, kw, first = parts.double().sum(0), torch.randn((nq,), generator=g), torch.randn((nk,), generator=g), torch.randn((T, nv), generator=g)
    cos = sin = None
    if dims:
        a = pos.double()[:, None] * P.yarn_frequencies(dims, 5000.0, None)[0]
        cos, sin = _f32(torch.cos(a)), _f32(torch.sin(a))
    pool = torch.full((1, n_pages, 2, kv_heads, page, row), 7.0, dtype=dtype, device=DEV)
    q, keep = torch.full((T, nq), 9.0, dtype=dtype, device=DEV), torch.full((T, nv), 9.0, device=DEV)
    ops.row_norm_qkv(_f32(parts), _f32(qw), _f32(kw), eps, cos, sin, ctx.positions, ctx.seg_of_token, q, KvLayerView(pool, 0, table), heads, dim, vdim, rt.status,
                     mix=None if mix is None else torch.tensor([mix], device=DEV), first=None if mix is None else _f32(first), keep=keep)
    tol = dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=2.0 ** -8, atol=1e-5)
    want_q = P.rotate((P.rms_unit(z[:, :nq], eps) * qw.double()).view(T, heads, dim), pos, rot, False).reshape(T, nq)
    want_k = P.rotate((P.rms_unit(z[:, nq:nq + nk], eps) * kw.double()).view(T, kv_heads, dim), pos, rot, False)
    own = z[:, nq + nk:]
    want_v = (own if mix is None else (1 - mix) * own + mix * first.double()).view(T, kv_heads, vdim)
    assert torch.allclose(q.cpu().double(), want_q, **tol) and torch.allclose(keep.cpu().double(), own, atol=1e-5)
    kept = pool.cpu().double()
    for t, p in enumerate(pos.tolist()):
        at = kept[0, perm[p // page], :, :, p % page]
        assert torch.allclose(at[0, :, :dim], want_k[t], **tol) and torch.allclose(at[1, :, :vdim], want_v[t], **tol)
    rt.check_status()


# ------------------------------------------------------------------------------------------ the matrix memory over portions and slots
SHORT = [[("a", 1), ("b", 2)], [("a", 1), ("b", 1)], [("a", 2)], [("a", 7), ("b", 6)], [("c", 1), ("a", 3)], [("c", 2), ("a", 9)], [("c", 11)], [("c", 1)], [("c", 1)]]
SLOTS = {"a": 0, "b": 2, "c": 2}      # b ends before c begins; c takes its slot, zeroed


def _long(C):
    return [[("a", 2 * C + 2), ("b", 3)], [("a", 1), ("b", C + 1)], [("a", 5 * C), ("b", 1)], [("c", C), ("a", 1)], [("c", 4 * C - 1), ("a", C + 7)], [("c", 1)]]


def _lens(plan):
    lens = {}
    for step in plan:
        for r, n in step:
            lens[r] = lens.get(r, 0) + n
    return lens


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("long_segments", [False, True])
@pytest.mark.parametrize("heads,dim,vdim,cap,i_bias,f_bias", [(3, 20, 12, 5.0, None, None), (5, 24, 24, 8.0, None, None), (2, 64, 128, 15.0, None, None), (1, 34, 6, 3.0, 9.0, None),
                                                              (2, 9, 33, 30.0, -25.0, 2.0), (2, 300, 31, 15.0, None, 12.0), (4, 16, 64, 12.0, -9.0, -9.0)])
def test_memory_over_portions_and_slots(dtype, long_segments, heads, dim, vdim, cap, i_bias, f_bias):
    """The mixer as a part, its state slots by hand: portions of 1, 2 and more tokens of three requests in two slots, or portions just below, at and
    above multiples of a chunk (and of the gates' 256 tokens), from zero and from earlier states, equal the plain recurrence over each whole
    sequence. Gates that stay at their caps, memories that keep everything or forget at once, input gates so low that the maximum follows the
    forget gates down from its start at zero (the bound e^(-m) then decides)."""
    from inference_bench_b200.cache.manager import StateView
    from inference_bench_b200.engine.runtime import Runtime
    from inference_bench_b200.kernels.ops import RECURRENCE_CHUNK
    from inference_bench_b200.parts.memory import MatrixMemory
    rt, W = Runtime(DEV, dtype=dtype), 64
    m = {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}
    w = _layer_tensors("mlstm", m, W, dim)
    for name, v in (("i", i_bias), ("f", f_bias)):
        if v is not None:
            w[f"l0.mix.{name}.b"] = torch.full_like(w[f"l0.mix.{name}.b"], v)
    part = MatrixMemory("l0.mix", W, heads, dim, vdim, cap, 1e-5)
    assert {s.name for s in part.weight_specs()} == {n for n in w if n.startswith("l0.mix")}
    part.bind({n: t.to(DEV) for n, t in w.items()}, rt)
    state, m_state = torch.zeros((3, heads, dim, vdim + 1), device=DEV), torch.zeros((3, heads), device=DEV)
    plan = _long(RECURRENCE_CHUNK) if long_segments else SHORT
    g = torch.Generator().manual_seed(W)
    x = {r: torch.randn((n, W), generator=g).to(torch.bfloat16) for r, n in _lens(plan).items()}
    want = {r: P.memory(t.double(), w, "l0.mix", m, 1e-5) for r, t in x.items()}
    with P.rounded():
        moved = {r: (P.memory(t.double(), w, "l0.mix", m, 1e-5) - want[r]).abs().amax(dim=1) / want[r].abs().max() for r, t in x.items()}
    at, tol = {}, 5e-5 if dtype == "float32" else 4e-2
    for step in plan:
        for r, _ in step:
            if r == "c" and r not in at:
                state[SLOTS[r]].zero_(), m_state[SLOTS[r]].zero_()
            at.setdefault(r, 0)
        ctx = _ctx(rt, [(at[r], n) for r, n in step], [SLOTS[r] for r, _ in step])
        xs = torch.cat([x[r][at[r]:at[r] + n] for r, n in step]).to(DEV, rt.act_dtype).contiguous()
        out = part.forward(ctx, xs, (StateView(state), StateView(m_state))).sum(0).cpu().double()
        o = 0
        for r, n in step:
            err = (out[o:o + n] - want[r][at[r]:at[r] + n]).abs().amax(dim=1) / want[r].abs().max()
            if dtype == "bfloat16":    # what rounding alone moves a row by in the plain form, times four, where that is more
                err = err * torch.clamp(tol / (4.0 * moved[r][at[r]:at[r] + n]), max=1.0)
            assert err.max().item() < tol, f"request {r} rows {at[r]}..{at[r] + n}: row {at[r] + int(err.argmax())} differs by {err.max().item():.2e}"
            o += n
            at[r] += n
    assert (state[1] == 0).all() and (m_state[1] == 0).all()      # nobody's slot
    rt.check_status()


def test_memory_states_and_maxima_are_the_scans(rt32):
    """What a segment leaves in its slot is the plain scan's running maximum, whichever kernel walked it: single tokens, short and long segments."""
    from inference_bench_b200.cache.manager import StateView
    from inference_bench_b200.parts.memory import MatrixMemory
    W, m = 48, {"heads": 3, "dim": 12, "vdim": 20, "gate_cap": 9.0}
    w = _layer_tensors("mlstm", m, W, 5)
    part = MatrixMemory("l0.mix", W, 3, 12, 20, 9.0, 1e-5)
    part.bind({n: t.to(DEV) for n, t in w.items()}, rt32)
    x = torch.randn((600, W), generator=torch.Generator().manual_seed(2)).to(torch.bfloat16)
    i, f = P.memory_gates(x.double(), w, "l0.mix", 9.0)
    top, tops = torch.zeros(3, dtype=F64), []
    for t in range(600):
        top = torch.maximum(f[t] + top, i[t])
        tops.append(top)
    for cuts in ((600,), (1, 599), (255, 1, 1, 2, 256, 85), (64, 65, 63, 408), tuple([1] * 30)):
        state, m_state, at = torch.zeros((2, 3, 12, 21), device=DEV), torch.zeros((2, 3), device=DEV), 0
        for n in cuts:
            part.forward(_ctx(rt32, [(at, n)], [1]), _f32(x[at:at + n]), (StateView(state), StateView(m_state)))
            at += n
            assert torch.allclose(m_state[1].cpu().double(), tops[at - 1], atol=1e-5), f"{cuts}: maximum after {at} tokens"


# ------------------------------------------------------------------------------------------ latent attention with a sink
@pytest.mark.parametrize("dtype,kernel", [("float32", "auto"), ("bfloat16", "auto"), ("bfloat16", "generic")])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank,q_rank,page,yarn", [(3, 12, 8, 20, 24, 40, 16, (4.0, 64, 8.0, 1.0)), (6, 32, 16, 48, 64, 96, 16, None), (2, 6, 4, 10, 18, 1, 8, None),
                                                                      (20, 16, 16, 16, 160, 32, 64, (8.0, 100, 4.0, 1.0)), (1, 64, 32, 32, 512, 64, 16, None), (40, 8, 16, 8, 32, 24, 16, None)])
def test_latent_attention_with_a_sink_over_a_paged_cache(dtype, kernel, heads, dim, rot, vdim, rank, q_rank, page, yarn):
    """The mixer as a part over its own cache: a prompt portion, portions down to two tokens and single tokens (whose keys are cut into slices), on
    shuffled pages, beside another request; sinks from far below the scores to above them; one far key made to stand out."""
    from inference_bench_b200.config.runtime_options import RuntimeOptions
    from inference_bench_b200.engine.runtime import Runtime
    from inference_bench_b200.kernels.ops import KvLayerView
    from inference_bench_b200.parts.latent import LatentAttention
    from inference_bench_b200.parts.standard import RotaryEmbedding
    rt, W = Runtime(DEV, options=RuntimeOptions(dtype=dtype, latent_attention=kernel)), 72
    r = {"dims": rot, "base": 1000.0}
    if yarn:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": 2.0 / math.sqrt(dim + rot), "rot": r}
    w = _layer_tensors("latent_attention", m, W, rank)
    w["l0.mix.sink"] = torch.linspace(-20.0, 9.0, heads).to(torch.bfloat16) if heads > 1 else torch.tensor([2.0], dtype=torch.bfloat16)
    part = LatentAttention("l0.mix", W, heads, dim, rot, vdim, rank, m["scale"], 1e-5, RotaryEmbedding(rot, 1000.0, "interleaved", yarn=yarn), q_rank=q_rank, sink=True)
    assert {s.name for s in part.weight_specs()} == {n for n in w if n.startswith("l0.mix")}
    part.bind({n: t.to(DEV) for n, t in w.items()}, rt)
    g = torch.Generator().manual_seed(rank)
    lens = {"a": 470, "b": 140}
    x = {k: torch.randn((n, W), generator=g).to(torch.bfloat16) for k, n in lens.items()}
    x["a"][468] = x["a"][17] * 3.0      # the row before the last asks for a key of the first pages
    want = {k: P.latent_attention(t.double(), w, "l0.mix", m, 1e-5) for k, t in x.items()}
    with P.rounded():
        moved = {k: (P.latent_attention(t.double(), w, "l0.mix", m, 1e-5) - want[k]).abs().amax(dim=1) / want[k].abs().max() for k, t in x.items()}
    n_pages = {k: -(-n // page) for k, n in lens.items()}
    perm = torch.randperm(sum(n_pages.values()), generator=g).to(torch.int32)
    tables = {"a": perm[:n_pages["a"]], "b": torch.cat([perm[n_pages["a"]:], torch.full((n_pages["a"] - n_pages["b"],), -1, dtype=torch.int32)])}
    pool = torch.full((1, len(perm), 1, 1, page, rank + rot), float("nan"), dtype=rt.act_dtype, device=DEV)
    at, tol = {"a": 0, "b": 0}, 3e-5 if dtype == "float32" else 3e-2
    steps = [[("a", 290)], [("a", 2), ("b", 1)], [("b", 127), ("a", 1)], [("a", 3)], [("b", 9), ("a", 168)]] + [[("a", 1), ("b", 1)]] * 3 + [[("a", 1)]] * 3
    for step in steps:
        ctx = _ctx(rt, [(at[k], n) for k, n in step])
        view = KvLayerView(pool, 0, torch.stack([tables[k] for k, _ in step]).contiguous().to(DEV))
        xs = torch.cat([x[k][at[k]:at[k] + n] for k, n in step]).to(DEV, rt.act_dtype).contiguous()
        out = part.forward(ctx, xs, view).sum(0).cpu().double()
        o = 0
        for k, n in step:
            err = (out[o:o + n] - want[k][at[k]:at[k] + n]).abs().amax(dim=1) / want[k].abs().max()
            if dtype == "bfloat16":
                err = err * torch.clamp(tol / (4.0 * moved[k][at[k]:at[k] + n]), max=1.0)
            assert err.max().item() < tol, f"request {k}, step {step}: row {at[k] + int(err.argmax())} differs by {err.max().item():.2e}"
            o += n
            at[k] += n
    assert at == lens
    rt.check_status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("slices", [1, 3])
def test_a_sink_far_above_every_score_leaves_almost_nothing(rt32, rt16, dtype, slices):
    """Sinks of 60 and -60 beside scores of order one: the output vanishes, or is the plain softmax's."""
    from inference_bench_b200.kernels import ops
    from inference_bench_b200.kernels.ops import KvLayerView
    rt = rt32 if dtype == torch.float32 else rt16
    g = torch.Generator().manual_seed(slices)
    H, rank, D, n = 2, 32, 48, 150
    q, rows = torch.randn((1, H, D), generator=g), torch.randn((160, D), generator=g).to(dtype)
    pool = rows.view(1, 10, 1, 1, 16, D).contiguous().to(DEV)
    view = KvLayerView(pool, 0, torch.arange(10, dtype=torch.int32, device=DEV).view(1, -1).contiguous())
    ctx = _ctx(rt, [(n - 1, 1)])
    out = torch.empty((1, H, rank), dtype=dtype, device=DEV)
    scratch = (torch.empty((H * slices * rank,), device=DEV), torch.empty((H * slices * 2,), device=DEV))
    sink = torch.tensor([60.0, -60.0], device=DEV)
    fn = ops.latent_attention if dtype == torch.float32 else ops.latent_attention_mma
    args = (_f32(q), view, ctx.positions, ctx.seg_of_token) + (() if dtype == torch.float32 else (None,))
    fn(*args, 0.2, out, rank, slices, 64 if slices > 1 else 1 << 30, scratch, rt.status, sink=sink)
    r = rows[:n].double()
    want = torch.softmax((q[0, 1].double() @ r.T) * 0.2, -1) @ r[:, :rank]
    got = out.cpu().double()[0]
    assert got[0].abs().max().item() < 1e-15 and torch.allclose(got[1], want, atol=1e-5 if dtype == torch.float32 else 2e-2)
    rt.check_status()


# ------------------------------------------------------------------------------------------ clamped feed-forwards
@pytest.mark.parametrize("T,inter,K", [(1, 64, 64), (1, 12288, 264), (8, 4096, 1024), (5, 200, 72), (17, 9472, 128), (33, 10304, 64), (64, 5000, 520), (100, 128, 64), (129, 520, 264), (700, 8192, 256),
                                       (2048, 384, 512), (2300, 1100, 72)])
@pytest.mark.parametrize("limit", [0.5, 7.0])
def test_product_with_clamped_pair(rt16, T, inter, K, limit):
    """The activation on the float32 accumulators in the tensor-core kernels' epilogues (or in the row-wise kernel where the k-range is cut)."""
    from inference_bench_b200.kernels import ops
    g = torch.Generator().manual_seed(T + inter + K)
    x = (torch.randn(T, K, generator=g) * 0.7).to(torch.bfloat16).to(DEV)
    lw = rt16.matrix((torch.randn(2 * inter, K, generator=g) * (3.0 / math.sqrt(K))).to(torch.bfloat16))
    act = rt16.gate_up_act(x, lw, ops.Clamp(torch.tensor([limit], device=DEV), 1.702))
    z = x.cpu().double() @ lw.weight.cpu().double().T
    want = P.clamped_glu(z[:, :inter], z[:, inter:], limit)
    assert ((act.cpu().double() - want).abs() <= 2.0 ** -8 * want.abs() + 2e-5 * want.abs().max()).all()
    rt16.check_status()


@pytest.mark.parametrize("dtype,how", [("float32", "auto"), ("bfloat16", "auto"), ("bfloat16", "mma"), ("bfloat16", "simt")])
@pytest.mark.parametrize("W,ff,experts,top,scale,shared", [(80, 24, 5, 2, 1.5, (48, 0.8)), (132, 36, 1, 1, 3.0, (20, 1.0)), (132, 28, 3, 1, 1.0, None), (192, 64, 16, 4, 2.5, (128, 2.0)),
                                                           (192, 128, 6, 6, 0.7, (128, 0.5)), (64, 40, 40, 3, 1.0, (8, 3.0))])
def test_experts_with_clamped_pairs(dtype, how, W, ff, experts, top, scale, shared):
    """Choice by corrected sigmoid scores, weights by the scores alone over their sum times a scale, experts and shared expert with limits of
    their own; one token to several hundred. Rows whose choice of the last expert is close are left out in bfloat16."""
    from inference_bench_b200.config.runtime_options import RuntimeOptions
    from inference_bench_b200.engine.runtime import Runtime
    from inference_bench_b200.parts.experts import RoutedExperts
    rt = Runtime(DEV, options=RuntimeOptions(dtype=dtype, expert_gemm=how))
    f = {"kind": "moe", "expert": {"ff": ff, "limit": 1.2}, "router": {"experts": experts, "top": top, "scale": scale},
         "shared": None if shared is None else {"ff": shared[0], "limit": shared[1]}}
    w = tg.tensors({"vocab": 8, "width": W, "layers": [{"type": "mlstm", "mixer": {"heads": 1, "dim": 4, "vdim": 4}, "mlp": f}]}, ff + experts)
    part = RoutedExperts("l0.mlp", W, ff, experts, top, route_scale=scale, renorm=True, shared_ff=shared[0] if shared else 0, score="sigmoid", correction="correction",
                         activation="clamped_swiglu", clamp=(1.2, 1.702), shared_limit=shared[1] if shared else 0.0)
    assert {s.name for s in part.weight_specs()} == {n for n in w if n.startswith("l0.mlp")}
    part.bind({n: t.to(DEV) for n, t in w.items()}, rt)
    g = torch.Generator().manual_seed(W)
    for T in (1, 3, 37, 70, 300):
        h = torch.randn((T, W), generator=g).to(torch.bfloat16)
        out = part.forward(_ctx(rt, [(0, T)]), h.to(DEV, rt.act_dtype).contiguous()).sum(0).cpu().double()
        want = P.experts_ff(h.double(), w, "l0.mlp", f)
        err = (out - want).abs().amax(1) / want.abs().max()
        if dtype == "bfloat16" and top < experts:
            z = torch.sort(torch.sigmoid(h.double() @ w["l0.mlp.router"].double().T) + w["l0.mlp.correction"].double(), descending=True).values
            err = err[(z[:, top - 1] - z[:, top]) > 1e-3]
        assert err.numel() == 0 or err.max().item() < (2e-5 if dtype == "float32" else 2e-2), f"{T} tokens: {err.max().item():.2e}"
    rt.check_status()


# ------------------------------------------------------------------------------------------ whole models
def _requests(name):
    vocab = tg.CONFIGS[name]["config"]["vocab"]
    return {r: traces.prompt(500 + i, n, vocab) for i, (r, n) in enumerate({"a": 150, "b": 1, "c": 23, "d": 64, "e": 97, "f": 2}.items())}


@pytest.fixture(scope="module")
def plain_logits(gdirs):
    return {name: {r: P.PlainGokosun(gdirs[name]).logits(t).numpy() for r, t in _requests(name).items()} for name in tg.CONFIGS}


@pytest.fixture(scope="module")
def rounded_logits(gdirs):
    with P.rounded():
        return {name: {r: P.PlainGokosun(gdirs[name]).logits(t).numpy() for r, t in _requests(name).items()} for name in tg.CONFIGS}


def _runner(model_dir, dtype, max_tokens, page_size, **kw):
    from inference_bench_b200.trace import build_runner
    return build_runner(model_dir, dtype, max_tokens, page_size=page_size, **kw)


def _compare(got, want_by_req, dtype, what, moved=None):
    """float32: every row. bfloat16: a row may differ by as much as TOLERANCE, or by four times what rounding alone moves it in the plain model
    (`moved`), except for one row in fifty (a router's close call), and half the rows are far closer (or within half as much again as the
    rounded plain model's)."""
    errs, over, plain = [], [], []
    for (r, pos), row in got.items():
        span = np.abs(want_by_req[r]).max()
        err = np.abs(row - want_by_req[r][pos]).max() / span
        errs.append(err)
        plain.append(0.0 if moved is None else np.abs(moved[r][pos] - want_by_req[r][pos]).max() / span)
        if not err <= max(TOLERANCE[dtype], 4.0 * plain[-1]):
            over.append((r, pos, float(err)))
    assert len(got) == sum(len(v) for v in want_by_req.values())
    assert len(over) <= (0 if dtype == "float32" else 0.02 * len(got)), f"{what}: rows over their limit: {over}"
    if dtype == "bfloat16":
        assert float(np.median(errs)) < max(BF16_MEDIAN, 1.5 * float(np.median(plain))), f"{what}: the median row differs by {np.median(errs):.2e} of max|logit|"
    return max(errs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tg.CONFIGS))
def test_layers_one_by_one(gdirs, name, dtype):
    """The residual stream after every layer against the plain model's, so that a wrong layer is named."""
    from inference_bench_b200.engine.step import StepEntry
    toks = _requests(name)["e"]
    plain = P.PlainGokosun(gdirs[name])
    want = plain.hidden_states(toks)
    with P.rounded():
        moved = plain.hidden_states(toks)
    runner = _runner(gdirs[name], dtype, 128, tg.CONFIGS[name]["page_size"])
    runner.cache.admit("x")
    layers = []
    runner.step([StepEntry("x", toks, list(range(len(toks))))], trace=layers)
    assert len(layers) == len(want) + 1
    for i, (g, w, r) in enumerate(zip(layers[1:], want, moved)):
        err = (g.cpu().double() - w).abs().amax(dim=1) / w.abs().max().item()
        if dtype == "bfloat16":     # what rounding alone moves a row by, times four, where that is more; a router's close call may fall the other way in a few rows
            err = err * torch.clamp(4e-2 / (4.0 * (r - w).abs().amax(dim=1) / w.abs().max()), max=1.0)
            err = err.sort().values[:int(0.9 * len(toks))]
        assert err.max().item() < (2e-5 if dtype == "float32" else 4e-2), f"{name}/{dtype}: the stream after layer {i} differs by {err.max().item():.2e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tg.CONFIGS))
@pytest.mark.parametrize("cut", ["whole", "tail", "portions", "mixed"])
def test_cut_matches_plain(gdirs, plain_logits, rounded_logits, name, dtype, cut):
    """Whole prompts; prompts then the last tokens one by one; portions down to two tokens; up to four live requests of unequal length in one
    batch with a pool that only holds what is live, so pages and slots are used again by later requests."""
    reqs = _requests(name)
    steps = {"whole": traces.whole, "tail": lambda r: traces.tail_one_by_one(r, tail=80), "portions": traces.portions, "mixed": traces.mixed}[cut](reqs)
    max_tokens = traces.max_live_tokens(steps)
    runner = _runner(gdirs[name], dtype, max_tokens, tg.CONFIGS[name]["page_size"], max_requests=4)
    got = traces.run_steps(runner, steps)
    worst = _compare(got, plain_logits[name], dtype, f"{name}/{dtype}/{cut}", rounded_logits[name] if dtype == "bfloat16" else None)
    runner.cache.check()
    assert runner.cache.used_pages() == [0] * len(runner.cache.groups)
    print(f"{name}/{dtype}/{cut}: worst {worst:.3e} of max|logit|, pool {max_tokens} tokens")


@pytest.mark.parametrize("name", ["A", "C"])
def test_a_request_alone_and_in_a_batch_give_the_same_float32_logits(gdirs, name):
    """The float32 path adds in one order whatever shares the step: a request beside three others of other lengths, on other pages and
    in another slot, gives the bits it gives alone."""
    from inference_bench_b200.engine.step import StepEntry
    reqs = _requests(name)
    runner = _runner(gdirs[name], "float32", 1024, 16, max_requests=4)
    runner.cache.admit("alone")
    alone = runner.step([StepEntry("alone", reqs["d"], [len(reqs["d"]) - 1])]).cpu()
    runner.cache.release("alone")
    for r in ("c", "f", "d", "a"):
        runner.cache.admit(r)
    rows = runner.step([StepEntry(r, reqs[r], [len(reqs[r]) - 1]) for r in ("c", "f", "d", "a")]).cpu()
    assert torch.equal(rows[2], alone[0])


# ------------------------------------------------------------------------------------------ weights made so that a fault shows
def _one(tmp_path, tag, kind, mixer, change=None, more=()):
    cfg = {"architecture": "Gokosun", "vocab": 64, "width": 40, "norm": {"eps": 1e-6}, "layers": [{"type": kind, "mixer": mixer, "mlp": None}, *more]}
    w = tg.tensors(cfg, 77)
    if change:
        change(w)
    return tg.write_folder(tmp_path / tag, cfg, w)


def _replay(model, toks, head, page, dtype="float32", chunk=None):
    """Logits of every position: a prompt of `head` tokens (in portions of `chunk`), then one by one."""
    from inference_bench_b200.engine.step import StepEntry
    runner = _runner(model, dtype, 64 * (-(-len(toks) // 64)), page)
    runner.cache.admit("x")
    rows, at = [], 0
    while at < len(toks):
        n = min(chunk or head, head - at) if at < head else 1
        rows.append(runner.step([StepEntry("x", toks[at:at + n], list(range(n)))]).cpu())
        at += n
    return torch.cat(rows).double()


@pytest.mark.parametrize("kind", ["latent_attention", "attention"])
@pytest.mark.parametrize("page", [8, 16])
def test_keys_far_away_and_at_page_borders(tmp_path, kind, page):
    """Queries and keys scaled until each softmax nearly picks one key: leaving out any one key (the first, at a page's edge, the token's own) would
    move rows by far more than the tolerance; the engine equals the plain model for whole prompts, portions and tokens decoded one by one."""
    if kind == "attention":
        mixer = {"heads": 2, "kv_heads": 1, "dim": 24, "vdim": 12, "scale": 1.5, "v_mix": False, "rot": {"base": 1e4, "dims": 4}}
    else:
        mixer = {"heads": 2, "dim": 20, "rot_dim": 4, "vdim": 12, "kv_rank": 28, "q_rank": 32, "scale": 1.5, "rot": {"base": 1e4, "dims": 4}}
    model = _one(tmp_path, kind, kind, mixer, lambda w: w["l0.mix.sink"].fill_(1.0) if kind == "latent_attention" else None)
    plain = P.PlainGokosun(model)
    toks = traces.prompt(11, 200, 64)
    for i, src in ((199, 0), (198, page - 1), (197, page), (150, 3 * page - 1), (151, 3 * page), (100, 0), (196, 195)):   # ask again for a token far back
        toks[i] = toks[src]
    want = plain.logits(toks)
    keep = P.causal_softmax
    for gone in (0, page - 1, page, 3 * page):
        def without(s, sink=None):
            s = s.clone()
            s[gone + 1:, gone] = -math.inf
            return keep(s, sink)
        try:
            P.causal_softmax = without
            diff = (plain.logits(toks) - want).abs().amax(dim=1) / want.abs().max()
        finally:
            P.causal_softmax = keep
        assert int((diff > 0.01).sum()) >= 1, f"a lost key {gone} would not show ({diff.max().item():.2e})"
    for head, chunk in ((200, None), (120, 7), (120, 2), (1, None)):
        err = (_replay(model, toks, head, page, chunk=chunk) - want).abs().amax(dim=1) / want.abs().max()
        assert err.max().item() < 2e-4, f"prompt of {head} in portions of {chunk}: {err.max().item():.2e} at position {int(err.argmax())}"


def test_the_first_token_counts_for_ever_and_long_decoding(tmp_path):
    """A memory whose first input gate is the largest and that forgets nothing: the first token still moves the logits 400 tokens on, through the
    chunked form and through 300 single tokens alike; the same for a latent layer behind it."""
    def keep_all(w):
        w["l0.mix.f.b"] = torch.full_like(w["l0.mix.f.b"], 11.0)
        w["l0.mix.i"] = torch.zeros_like(w["l0.mix.i"])
    mem = {"heads": 2, "dim": 16, "vdim": 8, "gate_cap": 20.0}
    lat = {"heads": 2, "dim": 6, "rot_dim": 4, "vdim": 10, "kv_rank": 12, "q_rank": 9, "scale": 0.3, "rot": {"base": 100.0, "dims": 4, "scaling": {"factor": 4.0, "original": 50, "fast": 4.0, "slow": 1.0}}}
    model = _one(tmp_path, "m", "mlstm", mem, keep_all, more=[{"type": "latent_attention", "mixer": lat, "mlp": None}])
    plain = P.PlainGokosun(model)
    toks = traces.prompt(12, 400, 64)
    want = plain.logits(toks)
    other = list(toks)
    other[0] = (toks[0] + 1) % 64
    assert ((plain.logits(other) - want)[-8:].abs().amax(dim=1) / want.abs().max()).median().item() > 1e-3
    for head in (400, 100):
        err = (_replay(model, toks, head, 16) - want).abs().amax(dim=1) / want.abs().max()
        assert err.max().item() < 1e-4, f"{head}: {err.max().item():.2e} at {int(err.argmax())}"


# ------------------------------------------------------------------------------------------ generation
@pytest.mark.parametrize("name", list(tg.CONFIGS))
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_engine(gdirs, name, graphs):
    """`Engine.generate`: the scheduler cuts prompts into portions, batches them beside decoded tokens, and decode steps run as captured
    graphs or not; float32 tokens equal the plain model's."""
    from inference_bench_b200 import Engine
    vocab = tg.CONFIGS[name]["config"]["vocab"]
    plain = P.PlainGokosun(gdirs[name])
    prompts = [traces.prompt(90 + i, n, vocab) for i, n in enumerate((5, 21, 40))]
    want = [plain.greedy(p, 7) for p in prompts]
    eng = Engine(gdirs[name], dtype="float32", max_ctx=128, page_size=tg.CONFIGS[name]["page_size"], use_graphs=graphs, prefill_chunk=9, max_batched_tokens=16)
    got = eng.generate(prompts, max_tokens=7)
    assert [r.tokens for r in got] == want
    assert eng.cache.used_pages() == [0] * len(eng.cache.groups)
    eng.cache.check()
    one = eng.generate(prompts[1], max_tokens=7)
    assert one.tokens == want[1]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sublayers_on_two_streams_give_the_bits_of_one(gdirs, dtype):
    """Captured decode steps with the feed-forward on a stream of its own: the logits of every step have the bits of the steps on one stream, for
    one request and for five (padded rows beside them)."""
    from inference_bench_b200 import Engine
    vocab = tg.CONFIGS["C"]["config"]["vocab"]
    prompts = [traces.prompt(30 + i, n, vocab) for i, n in enumerate((9, 40, 3, 70, 17))]
    out = []
    for side in (True, False):
        eng = Engine(gdirs["C"], dtype=dtype, max_ctx=256, page_size=16, options={"side_stream": side})
        tokens = [r.tokens for r in eng.generate(prompts, max_tokens=24)] + [eng.generate(prompts[1], max_tokens=24).tokens]
        out.append((tokens, eng.executor.last_logits.clone() if eng.executor.last_logits is not None else None))
    assert out[0][0] == out[1][0]
    assert out[0][1] is None or torch.equal(out[0][1], out[1][1])


def test_generation_in_bfloat16_runs_and_long_decoding_stays_close(gdirs):
    from inference_bench_b200 import Engine
    name = "C"
    vocab = tg.CONFIGS[name]["config"]["vocab"]
    plain = P.PlainGokosun(gdirs[name])
    prompt = traces.prompt(5, 12, vocab)
    eng = Engine(gdirs[name], dtype="bfloat16", max_ctx=256, page_size=16)
    got = eng.generate(prompt, max_tokens=120).tokens
    assert len(got) == 120
    lg = plain.logits(prompt + got)     # teacher-forced on the engine's own tokens, the plain model ranks every chosen token near the top
    span = float(lg.max() - lg.min())
    below = [float(lg[len(prompt) + i - 1].max() - lg[len(prompt) + i - 1][tok]) / span for i, tok in enumerate(got)]
    assert all(math.isfinite(b) for b in below) and max(below) < 0.2
    assert sum(b > 0.03 for b in below) <= 0.1 * len(got)


def test_trace_replay_program_and_command_line(gdirs, tmp_path):
    """bin/trace_run as a subprocess fed JSON steps (a mixed trace, float32), and `run` and `spec` of the command line, on a model folder
    of this architecture: nothing in them names an architecture."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    name = "A"
    vocab = tg.CONFIGS[name]["config"]["vocab"]
    reqs = {r: traces.prompt(900 + i, n, vocab) for i, (r, n) in enumerate({"a": 70, "b": 9, "c": 33, "d": 64, "e": 2}.items())}
    steps = traces.mixed(reqs, seed=5)
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(gdirs[name]), "--dtype", "float32", "--out", str(out),
                           "--max-tokens", str(traces.max_live_tokens(steps))],
                          input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    plain = P.PlainGokosun(gdirs[name])
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
    p = subprocess.run([sys.executable, "-m", "inference_bench_b200", "run", "--model", str(gdirs[name]), "--prompt-len", "12", "--max-tokens", "5", "--json",
                        "--dtype", "float32", "--max-ctx", "64"], capture_output=True, text=True, env=env, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    r = json.loads(p.stdout)
    from inference_bench_b200.cli import _synthetic_prompt
    assert r["prompt_tokens"] == 12 and r["tokens"] == plain.greedy(_synthetic_prompt(12, vocab), 5)
    p = subprocess.run([sys.executable, "-m", "inference_bench_b200", "spec", "--model", str(gdirs[name])], capture_output=True, text=True, env=env)
    assert p.returncode == 0 and json.loads(p.stdout)["layers"][2]["mixer"]["gate_cap"] == 5.0
