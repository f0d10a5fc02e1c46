"""Tile and split choice for the tcgen05 matrix product, and its launch.

The kernel puts 128 weight rows and `bn` tokens in a CTA. Few tokens leave few CTAs, so the k-range
of a tile is then split over several CTAs, each writing its own float32 partial; the consumer kernel
adds the partials in a fixed order, so results are reproducible. The choice depends only on the
sizes of the product (T, N, K), never on which requests make up the batch.
"""
from __future__ import annotations

import ctypes as C
import functools
from typing import Optional

import torch

from . import lib as L
from . import ops

FITTED_SM_COUNT = 148   # the part the cost model below was fitted on; every function takes the running device's count as an argument
TOKEN_TILES = (16, 32, 64, 128, 256)

L.register("ib_gemm_tcgen05", [L._p, L._p, L._p, L._i, L._i, L._i, L._i, L._i, L._i, L._p, L._p])
L.register("ib_gemm_swiglu_tcgen05", [L._p, L._p, L._p, L._i, L._i, L._i, L._i, L._i, L._p, L._f, L._p, L._p])
L.register("ib_gemm_tcgen05_2cta", [L._p, L._p, L._p, L._i, L._i, L._i, L._p, L._p])
L.register("ib_gemm_swiglu_tcgen05_2cta", [L._p, L._p, L._p, L._i, L._i, L._i, L._p, L._f, L._p, L._p])
L.register("ib_gemm_xielu_tcgen05", [L._p, L._p, L._p, L._i, L._i, L._i, L._i, L._i, L._p, L._p, L._p])
L.register("ib_gemm_xielu_tcgen05_2cta", [L._p, L._p, L._p, L._i, L._i, L._i, L._p, L._p, L._p])
L.register("ib_gemm_relu2_tcgen05", [L._p, L._p, L._p, L._i, L._i, L._i, L._i, L._i, L._p, L._p])
L.register("ib_gemm_relu2_tcgen05_2cta", [L._p, L._p, L._p, L._i, L._i, L._i, L._p, L._p])
L.register("ib_gemm_tcgen05_2cta_add", [L._p, L._p, L._p, L._i, L._i, L._i, L._p, L._p])
L.register("ib_gemm_qkv_tcgen05_2cta", [L._p, L._p, L._i, L._i, L._p, L._p, L._f, L._p, L._p, L._p, L._p, L._p, C.POINTER(L.KvView), L._i, L._i, L._p, L._p])

L.register("ib_gemm_grouped_tcgen05", [L._p, L._p, L._p, L._i, L._i, L._i, L._i, L._p, L._p, L._i, L._p, L._p])
L.register("ib_gemm_parts_tcgen05", [L._p, L._p, L._p, L._i, L._i, L._i, L._i, L._i, L._i, L._p, L._p])
L.register("ib_gemm_grouped_relu2_tcgen05", [L._p, L._p, L._p, L._i, L._i, L._i, L._i, L._p, L._p, L._i, L._p, L._p])
L.register("ib_gemm_grouped_swiglu_tcgen05", [L._p, L._p, L._p, L._i, L._i, L._i, L._i, L._p, L._p, L._i, L._p, L._f, L._p, L._p])

# Runtime options that steer the choice (config/runtime_options.py): `pair_min_tokens` (129: the fused gate/up product runs on the
# persistent CTA-pair kernel, csrc/gemm_tcgen05_2cta.cu, from here on whatever its size), `pair_always_tokens` (2,048: every
# product from here on; between the two, `plan` decides by its cost model) and `fuse_qkv_epilogue`.


def supports(k: int) -> bool:
    return k % 8 == 0


@functools.lru_cache(maxsize=4096)
def choose(T: int, N: int, K: int, allow_split: bool = True, sm_count: int = FITTED_SM_COUNT) -> tuple[int, int, bool]:
    """(tokens per CTA, k-splits, wide) for up to 128 tokens: the smallest token tile that holds them, and the
    k-range split over CTAs until the GPU is full."""
    if T > 128:
        raise ValueError(f"choose is for up to 128 tokens, got {T}: see plan")
    ktiles = -(-K // 64)
    bn = next(b for b in TOKEN_TILES if T <= b)
    tiles = -(-N // 128)
    slots = sm_count * (2 if bn <= 64 else 1)      # CTAs resident at once (two per SM for the small token tiles)
    splits = 1
    if allow_split and tiles < slots:
        splits = max(1, min(slots // tiles, ktiles // 4, 16))
        per = -(-ktiles // splits)
        splits = -(-ktiles // per)  # no empty split
    return bn, splits, False


# Cost model for 129 to 2,048 tokens, fitted to timings of every variant below on the layer shapes of Qwen3-0.6B, 8B,
# 14B and 32B at 160 to 1,536 tokens (the variant it picks is within 5 % of the fastest on all of them, 0.2 % on
# average). A variant's time is waves of CTAs (or CTA pairs) times the longer of a CTA's MMA time and its copy time,
# plus a fixed cost, plus the traffic of split-K partial sums. Units: FLOP/us, bytes/us, us.
_MID = dict(rate=4.015e6, cap=250e3, t0=4.36, partial_bw=3.455e6, pair_rate=5.446e6, hbm=8.0e6, pair_cap=188e3,
            speed={(256, True): 1.0, (256, False): 0.982, (128, True): 0.895, (128, False): 0.956})


def single_variants(T: int, N: int, K: int, sm_count: int = FITTED_SM_COUNT, allow_split: bool = True):
    """The forms of the single-CTA kernel that `plan` weighs for more than 128 tokens: (tokens per CTA, k-splits, wide)."""
    ktiles = -(-K // 64)
    for bn in (128, 256):
        for wide in (False, True):
            for sp in ((1, 2, 3, 4, 6) if allow_split else (1,)):
                per = -(-ktiles // sp)
                if sp > max(1, ktiles // 4) or -(-ktiles // per) != sp:   # at least four k-tiles a split, and none empty
                    continue
                ctas = -(-N // (256 if wide else 128)) * -(-T // bn) * sp
                if sp > 1 and ctas > 4 * sm_count:
                    continue
                yield bn, sp, wide


@functools.lru_cache(maxsize=4096)
def plan_costs(T: int, N: int, K: int, sm_count: int = FITTED_SM_COUNT, allow_split: bool = True) -> tuple:
    """(expected us of the CTA-pair kernel, expected us of the best single-CTA form, that form) for 129 <= T < 2048.
    allow_split=False leaves out the forms that cut the k-range (for a caller that wants one finished product)."""
    m = _MID
    tiles = -(-N // 256) * -(-T // 256)
    active = min(tiles, sm_count // 2) * 2
    pair = -(-tiles // (sm_count // 2)) * max(256 * 256 * K * 2 / (2 * m["pair_rate"]), 256 * K * 2 / min(m["pair_cap"], m["hbm"] / active)) + m["t0"]
    best = (float("inf"), None)
    ktiles = -(-K // 64)
    for bn, sp, wide in single_variants(T, N, K, sm_count, allow_split):
        rows = 256 if wide else 128
        ctas = -(-N // rows) * -(-T // bn) * sp
        kc = -(-ktiles // sp) * 64
        mma = rows * bn * kc * 2 / (m["rate"] * m["speed"][(bn, wide)])
        copy = (rows + min(bn, T)) * kc * 2 / min(m["cap"], m["hbm"] / min(ctas, sm_count))
        t = -(-ctas // sm_count) * max(mma, copy) + m["t0"] + (sp * T * N * 4 / m["partial_bw"] if sp > 1 else 0.0)
        if t < best[0]:
            best = (t, (bn, sp, wide))
    return pair, best[0], best[1]


def plan(T: int, N: int, K: int, sm_count: int = FITTED_SM_COUNT, allow_split: bool = True) -> tuple:
    """For 129 <= T < 2048: ("pair",) or ("single", tokens per CTA, k-splits, wide), whichever the cost model
    expects to be faster. Depends on the sizes (and the device's SM count) only."""
    pair, single, form = plan_costs(T, N, K, sm_count, allow_split)
    return ("pair",) if pair <= single else ("single",) + form


def qkv_in_epilogue(rt, T: int, N: int, K: int) -> bool:
    """Whether the q/k/v projection of T tokens runs as the CTA-pair kernel with the q/k norm, the rotation and the
    cache write in its epilogue: from 2,048 tokens always; from 129 when that is expected to take no longer than the
    best plain product followed by the kernel it saves (about 3 us + 20 ns a token inside a step)."""
    if not rt.options.qkv_epilogue or T <= 128:
        return False
    if T >= rt.options.pair_always_tokens:
        return True
    pair, single, _ = plan_costs(T, N, K, rt.sm_count)
    return pair <= single + 3.0 + 0.02 * T


def balanced_portion(matrices, nominal: int = 2048, sm_count: int = FITTED_SM_COUNT) -> int:
    """A prompt-portion size near `nominal` (a multiple of 256 between 3/4 and 5/4 of it) whose 256 x 256 tiles fill
    whole rounds of the CTA pairs best, for the [N, K] matrices of a layer: the time a token costs is taken as the sum
    over the matrices of K x rounds x 74 tiles / tokens. The CTA-pair products work in rounds of 74 tiles, and a portion
    that ends in a nearly empty round pays for it (measured: 14B shape 45.2 k tok/s at 1,792 tokens against 41.3 k at
    2,048; 32B 19.0 against 18.1 k; 8B 80.8 k at 2,304 against 79.9 k). Ties go to the size nearest to `nominal`."""
    pairs = sm_count // 2
    best = None
    for T in range(max(256, nominal * 3 // 4 // 256 * 256), nominal * 5 // 4 + 1, 256):
        cost = sum(k * -(-(-(-n // 256) * -(-T // 256)) // pairs) for n, k in matrices) / T
        key = (cost, abs(T - nominal), -T)
        if best is None or key < best[0]:
            best = (key, T)
    return best[1] if best else nominal


def gemm(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, bn: int, splits: int, status: torch.Tensor, wide: bool = False) -> None:
    """out [splits, T, N] float32 = per-split partial products of x [T, K] and w [N, K] (bfloat16).
    wide: 256 rows of w per CTA instead of 128 (token tiles of 128 or 256 only)."""
    T, K = x.shape
    N = w.shape[0]
    ops._check("x", x, torch.bfloat16)
    ops._check("w", w, torch.bfloat16, (N, K))
    ops._check("out", out, torch.float32, (splits, T, N))
    L.call("ib_gemm_tcgen05", x.data_ptr(), w.data_ptr(), out.data_ptr(), T, N, K, bn, splits, 1 if wide else 0, status.data_ptr(), ops._stream())


def gemm_pair(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, status: torch.Tensor, add: bool = False) -> None:
    """out [T, N] float32 = x [T, K] w[N, K]^T on CTA pairs (256 x 256 tiles, persistent); with `add`
    the product is added to what out holds."""
    T, K = x.shape
    N = w.shape[0]
    ops._check("x", x, torch.bfloat16)
    ops._check("w", w, torch.bfloat16, (N, K))
    ops._check("out", out, torch.float32, (T, N))
    L.call("ib_gemm_tcgen05_2cta_add" if add else "ib_gemm_tcgen05_2cta", x.data_ptr(), w.data_ptr(), out.data_ptr(), T, N, K, status.data_ptr(), ops._stream())


def gemm_qkv_pair(x: torch.Tensor, w: torch.Tensor, q_out: torch.Tensor, kv: "ops.KvLayerView", heads: int, q_norm_w: Optional[torch.Tensor],
                  k_norm_w: Optional[torch.Tensor], eps: float, cos: Optional[torch.Tensor], sin: Optional[torch.Tensor], positions: torch.Tensor,
                  seg_of_token: torch.Tensor, write_kv: bool, status: torch.Tensor) -> None:
    """q_out [T, heads * 128] bfloat16 and the paged cache from x [T, K] and w [(heads + 2 kv_heads) * 128, K]: the
    projection, the per-head norms, the rotation and the cache write in one kernel (csrc/gemm_tcgen05_2cta.cu)."""
    T, K = x.shape
    view = kv.c_view()
    if view.head_dim != 128 or (cos is not None and cos.shape[1] != 64):
        raise L.KernelError(f"gemm_qkv_pair: head size {view.head_dim} with a rotation over {None if cos is None else 2 * cos.shape[1]} values (128 and 128 or none)")
    N = (heads + 2 * view.kv_heads) * 128
    ops._check("x", x, torch.bfloat16)
    ops._check("w", w, torch.bfloat16, (N, K))
    ops._check("q_out", q_out, torch.bfloat16, (T, heads * 128))
    ops._check("positions", positions, torch.int32, (T,))
    ops._check("seg_of_token", seg_of_token, torch.int32, (T,))
    for name, v in (("q_norm", q_norm_w), ("k_norm", k_norm_w)):
        if v is not None:
            ops._check(name, v, torch.float32, (128,))
    if cos is not None:
        ops._check("cos", cos, torch.float32, (T, 64))
        ops._check("sin", sin, torch.float32, (T, 64))
    L.call("ib_gemm_qkv_tcgen05_2cta", x.data_ptr(), w.data_ptr(), T, K, ops._ptr(q_norm_w), ops._ptr(k_norm_w), float(eps), ops._ptr(cos), ops._ptr(sin),
           positions.data_ptr(), seg_of_token.data_ptr(), q_out.data_ptr(), C.byref(view), 1 if write_kv else 0, heads, status.data_ptr(), ops._stream())


def linear(rt, x: torch.Tensor, lw, allow_split: bool = True, add_to: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    T = x.shape[0]
    how = ("pair",) if T >= rt.options.pair_always_tokens else (plan(T, lw.n, lw.k, rt.sm_count, allow_split) if T > 128 else None)
    if how is not None and how[0] == "single":
        _, bn, splits, wide = how
        out = rt.empty((splits, T, lw.n), torch.float32)
        gemm(x, lw.weight, out, bn, splits, rt.status, wide)
        return out
    if how is not None:
        if add_to is not None:
            gemm_pair(x, lw.weight, add_to, rt.status, add=True)
            return None
        out = rt.empty((1, T, lw.n), torch.float32)
        gemm_pair(x, lw.weight, out[0], rt.status)
        return out
    bn, splits, wide = choose(T, lw.n, lw.k, allow_split, rt.sm_count)
    out = rt.empty((splits, T, lw.n), torch.float32)
    gemm(x, lw.weight, out, bn, splits, rt.status, wide)
    return out


PAIR_SWIGLU_MIN_TILES = 40   # 256-column blocks of the intermediate size from which the CTA-pair kernel takes the fused gate/up product of 33 to 128 tokens


HALF_SWIGLU_MIN_CTAS = 148   # CTAs (intermediate size / 64) from which the form with gate and up rows in one accumulator is used
HALF_SWIGLU_MAX_TOKENS = 64   # ... and up to how many tokens (at 64 tokens 0.7 % of a batch-64 decode step faster than the CTA-pair form, Qwen3-8B shape)


def swiglu_supported(T: int, k: int, inter: int = 0) -> bool:
    """Whether the gate/up product applies the activation in its epilogue: from 65 tokens always; from 33 where the
    intermediate size gives the CTA-pair kernel 40 tiles or more (measured 8 to 10 % faster there than the split-K
    product followed by the SiLU-mul kernel, at the 8B, 14B and 32B shapes; slower at the 0.6B shape); up to 64 tokens
    in the form that puts 64 gate rows and their 64 up rows into one accumulator, where the intermediate size is a
    multiple of 64 and gives every SM a CTA (a smaller one goes through the split-K product and the SiLU-mul kernel,
    which then fill the GPU better)."""
    if not supports(k):
        return False
    if half_swiglu(T, inter):
        return True
    return T > 64 or (T > 32 and -(-inter // 256) >= PAIR_SWIGLU_MIN_TILES)


def half_swiglu(T: int, inter: int) -> bool:
    """Whether the fused gate/up product of T tokens takes the form with 64 gate rows and 64 up rows in one accumulator."""
    return T <= HALF_SWIGLU_MAX_TOKENS and inter % 64 == 0 and inter // 64 >= HALF_SWIGLU_MIN_CTAS


def gemm_swiglu(x: torch.Tensor, w_gate_up: torch.Tensor, act: torch.Tensor, status: torch.Tensor, bn: int | None = None, pair_min_tokens: int = 129,
                half: bool | None = None, clamp: Optional["ops.Clamp"] = None) -> None:
    """act [T, I] bfloat16 = silu(x gate^T) * (x up^T) (or the clamped pair) with w_gate_up [2I, K] = gate rows then up rows."""
    T, K = x.shape
    I = w_gate_up.shape[0] // 2
    ops._check("x", x, torch.bfloat16)
    ops._check("w_gate_up", w_gate_up, torch.bfloat16, (2 * I, K))
    ops._check("act", act, torch.bfloat16, (T, I))
    if bn is None and (half_swiglu(T, I) or (T <= 32 and I % 64 == 0)):
        bn, half = (16 if T <= 16 else 32 if T <= 32 else 64), True
    if half is None:
        half = bn in (16, 32)
    if bn is None and (T >= pair_min_tokens or (T > 32 and -(-I // 256) >= PAIR_SWIGLU_MIN_TILES)):
        L.call("ib_gemm_swiglu_tcgen05_2cta", x.data_ptr(), w_gate_up.data_ptr(), act.data_ptr(), T, I, K, *ops._clamp_args(clamp), status.data_ptr(), ops._stream())
        return
    if bn is None:
        bn = 64 if T <= 64 else (128 if T <= 128 else 256)
    L.call("ib_gemm_swiglu_tcgen05", x.data_ptr(), w_gate_up.data_ptr(), act.data_ptr(), T, I, K, bn, 1 if half else 0, *ops._clamp_args(clamp), status.data_ptr(), ops._stream())


ACT_MIN_ROW_BLOCKS = 32   # 128-row blocks of the matrix from which up to 128 tokens keep the whole k-range in one CTA (that many CTAs fill the memory system)


def act_in_epilogue(T: int, N: int, K: int, sm_count: int = FITTED_SM_COUNT) -> bool:
    """Whether the product of T tokens with an [N, K] matrix applies an activation (xIELU, squared ReLU) in its epilogue: above 128 tokens always; up to
    128 when the matrix has enough row blocks to fill the GPU without cutting the k-range (otherwise the k-range is split over CTAs and
    a row-wise kernel adds the partial sums). A function of the sizes only."""
    if not supports(K):
        return False
    return T > 128 or -(-N // 128) >= ACT_MIN_ROW_BLOCKS or choose(T, N, K, True, sm_count)[1] == 1


def gemm_act(rt, x: torch.Tensor, lw, kind: str, act: torch.Tensor, pq: Optional[torch.Tensor] = None) -> None:
    """act [T, N] bfloat16 = activation of x w^T: kind "xielu" with pq = (p, q) float32 on the device, or "relu2" (max(z, 0)^2); the kernel's form is
    chosen like `linear`'s, without cutting the k-range."""
    T, K = x.shape
    ops._check("x", x, torch.bfloat16)
    ops._check("w", lw.weight, torch.bfloat16, (lw.n, K))
    ops._check("act", act, torch.bfloat16, (T, lw.n))
    extra = ()
    if kind == "xielu":
        ops._check("pq", pq, torch.float32, (2,))
        extra = (pq.data_ptr(),)
    elif kind != "relu2":
        raise L.KernelError(f"gemm_act: activation {kind!r} is not known (xielu, relu2)")
    how = ("pair",) if T >= rt.options.pair_always_tokens else (plan(T, lw.n, K, rt.sm_count, False) if T > 128 else None)
    if how is not None and how[0] == "pair":
        L.call(f"ib_gemm_{kind}_tcgen05_2cta", x.data_ptr(), lw.weight.data_ptr(), act.data_ptr(), T, lw.n, K, *extra, rt.status.data_ptr(), ops._stream())
        return
    bn, _, wide = how[1:] if how is not None else choose(T, lw.n, K, False, rt.sm_count)
    L.call(f"ib_gemm_{kind}_tcgen05", x.data_ptr(), lw.weight.data_ptr(), act.data_ptr(), T, lw.n, K, bn, 1 if wide else 0, *extra, rt.status.data_ptr(), ops._stream())


# ---------------------------------------------------------------- products on regrouped rows (routed experts)
def grouped_token_tile(rows: int, groups: int, inter: int = 0, sm_count: int = FITTED_SM_COUNT) -> int:
    """Tokens per CTA for a product on `rows` regrouped rows of `groups` experts: the smallest tile that holds an expert's average share,
    up to 128; 256 where the experts' shares are larger and tiles of 256 still give every SM two CTAs (measured alone, 2,048 tokens: 64
    experts of 1,408 x 2,048 with 6 a token 421 against 468 us; 16 experts of 1,024 x 1,024 with 2 a token 87 against 83 us). A function of
    the sizes only."""
    avg = -(-rows // groups)
    if avg <= 128:
        return 16 if avg <= 16 else 32 if avg <= 32 else 64 if avg <= 64 else 128
    ctas = (rows // 256 + groups // 2) * max(1, -(-inter // 128))
    return 256 if ctas >= 2 * sm_count else 128


def grouped_supported(k: int, inter: int, bn: int, gated: bool = True) -> bool:
    """Whether the tcgen05 kernel takes the experts' two products: inner sizes that are multiples of 8, and for gated experts and tiles of 16 or
    32 tokens (64 gate rows and their up rows in one accumulator) an expert size that is a multiple of 64."""
    return k % 8 == 0 and inter % 8 == 0 and (not gated or bn >= 64 or inter % 64 == 0)


def gemm_grouped(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, bn: int, offsets: torch.Tensor, tiles: torch.Tensor, status: torch.Tensor) -> None:
    """out [R, N] float32 = per expert w[e] x[r] for the regrouped rows x [R, K] (expert e's rows: offsets[e] .. offsets[e + 1]); w [E, N, K];
    tiles: first token tile of `bn` rows of every expert, then their number (`ops.moe_sort` with tile_rows=bn)."""
    R, K = x.shape
    E, N, _ = w.shape
    ops._check("x", x, torch.bfloat16)
    ops._check("w", w, torch.bfloat16, (E, N, K))
    ops._check("out", out, torch.float32, (R, N))
    L.call("ib_gemm_grouped_tcgen05", x.data_ptr(), w.data_ptr(), out.data_ptr(), R, N, K, bn, offsets.data_ptr(), tiles.data_ptr(), E, status.data_ptr(), ops._stream())


PARTS_MAX_TOKENS = 128   # up to here several products of one shape run as one launch; above, each product fills the GPU by itself


def gemm_parts(rt, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x [parts, T, K], w [parts, N, K] (bfloat16) -> float32 partial sums [P, parts, T, N] of every part's product with its own matrix, in one launch."""
    parts, T, K = x.shape
    N = w.shape[1]
    ops._check("x", x, torch.bfloat16)
    ops._check("w", w, torch.bfloat16, (parts, N, K))
    bn, splits, _ = choose(T, parts * N, K, True, rt.sm_count)
    out = rt.empty((splits, parts, T, N), torch.float32)
    L.call("ib_gemm_parts_tcgen05", x.data_ptr(), w.data_ptr(), out.data_ptr(), parts, T, N, K, bn, splits, rt.status.data_ptr(), ops._stream())
    return out


def gemm_grouped_relu2(x: torch.Tensor, w: torch.Tensor, act: torch.Tensor, bn: int, offsets: torch.Tensor, tiles: torch.Tensor, status: torch.Tensor) -> None:
    """act [R, N] bfloat16 = max(w[e] x[r], 0)^2 for the regrouped rows; arguments as for `gemm_grouped`."""
    R, K = x.shape
    E, N, _ = w.shape
    ops._check("x", x, torch.bfloat16)
    ops._check("w", w, torch.bfloat16, (E, N, K))
    ops._check("act", act, torch.bfloat16, (R, N))
    L.call("ib_gemm_grouped_relu2_tcgen05", x.data_ptr(), w.data_ptr(), act.data_ptr(), R, N, K, bn, offsets.data_ptr(), tiles.data_ptr(), E, status.data_ptr(), ops._stream())


def gemm_grouped_swiglu(x: torch.Tensor, w_gate_up: torch.Tensor, act: torch.Tensor, bn: int, offsets: torch.Tensor, tiles: torch.Tensor, status: torch.Tensor,
                        clamp: Optional["ops.Clamp"] = None) -> None:
    """act [R, I] bfloat16 = silu(gate_e x) * (up_e x) (or the clamped pair, one limit an expert) per expert, w_gate_up [E, 2 I, K] = every expert's gate rows then its up rows."""
    R, K = x.shape
    E, I2, _ = w_gate_up.shape
    ops._check("x", x, torch.bfloat16)
    ops._check("w_gate_up", w_gate_up, torch.bfloat16, (E, I2, K))
    ops._check("act", act, torch.bfloat16, (R, I2 // 2))
    L.call("ib_gemm_grouped_swiglu_tcgen05", x.data_ptr(), w_gate_up.data_ptr(), act.data_ptr(), R, I2 // 2, K, bn, offsets.data_ptr(), tiles.data_ptr(), E,
           *ops._clamp_args(clamp, E), status.data_ptr(), ops._stream())
