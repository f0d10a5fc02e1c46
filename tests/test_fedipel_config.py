"""Fedipel without a device: the configuration's reader and its refusals, the plan (schedule, shared caches, tensor names and shapes), the
pages a window with kept first positions holds, and the plain implementation's own pieces on cases small enough to do by hand."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_fedipel as P
import tiny_fedipel as tf
from inference_bench_b200.cache.manager import CacheManager
from inference_bench_b200.config import ConfigError
from inference_bench_b200.config.fedipel import FedipelConfig
from inference_bench_b200.engine.model import plan_from_config
from inference_bench_b200.parts.base import FixedState, PagedKV, Several
from inference_bench_b200.parts.decoder import Decoder
from inference_bench_b200.weights.loader import WeightError, WeightStore
from inference_bench_b200.weights.random_init import write_random_model


@pytest.mark.parametrize("name", list(tf.CONFIGS))
def test_config_round_trip_and_plan(name):
    raw = tf.CONFIGS[name]["config"]
    cfg = FedipelConfig.from_dict(raw)
    assert FedipelConfig.from_dict(cfg.to_dict()) == cfg
    _, plan = plan_from_config(raw)
    dec = Decoder(plan)
    specs = {s.name: s for s in dec.weight_specs()}
    made = tf.tensors(raw, 1, rank=7)                     # the decay's inner size is the tensors' own
    assert set(specs) == set(made) and all(specs[n].fits(tuple(made[n].shape)) for n in made)
    assert [e.layer for e in plan.schedule] == list(range(len(raw["layers"])))
    for l, e, need in zip(raw["layers"], plan.schedule, dec.cache_needs()):
        m = l["mixer"]
        if l["type"] == "retention":
            assert need == FixedState((m["heads"], m["dim"], m["vdim"]), torch.float32)
        elif l["type"] == "wkv":
            assert need == Several((FixedState((m["heads"], m["dim"], m["dim"]), torch.float32), FixedState((raw["width"],), torch.float32)))
        elif m.get("kv_from") is not None:
            assert need is None and e.cache_of == m["kv_from"]
        else:
            assert isinstance(need, PagedKV) and need.kv_heads == m["kv_heads"] and need.head_dim == max(2 * m["dim"], m["vdim"])


def test_a_cache_holds_what_every_reader_sees():
    """Layer 0 of A sees 9 positions back and keeps 3; its readers see 40 back and keep 1, and see 5 back and keep 19."""
    _, plan = plan_from_config(tf.CONFIGS["A"]["config"])
    need = Decoder(plan).cache_needs()[0]
    assert (need.window, need.keep_first) == (40, 19)
    raw = copy.deepcopy(tf.CONFIGS["A"]["config"])
    raw["layers"][2]["mixer"]["mask"] = None              # a reader without a window: everything stays
    need = Decoder(plan_from_config(raw)[1]).cache_needs()[0]
    assert (need.window, need.keep_first) == (None, 0)


@pytest.mark.parametrize("path,value,words", [
    (("layers", 0, "type"), "mamba2", "not supported"),
    (("layers", 0, "mixer", "kv_heads"), 3, "multiple"),
    (("layers", 0, "mixer", "rot", "dims"), 7, "even"),
    (("layers", 0, "mixer", "rot", "dims"), 18, "at most dim"),
    (("layers", 0, "mixer", "dim"), 130, "at most 256"),
    (("layers", 0, "mixer", "mask", "size"), 0, "positive"),
    (("layers", 0, "mixer", "mask", "keep_first"), -1, "not negative"),
    (("layers", 2, "mixer", "kv_from"), 1, "earlier attention layer"),
    (("layers", 2, "mixer", "kv_from"), 2, "earlier attention layer"),
    (("layers", 4, "mixer", "kv_from"), 2, "no keys and values of its own"),
    (("layers", 2, "mixer", "vdim"), 16, "differ"),
    (("layers", 2, "mixer", "rot", "base"), 10.0, "differ"),
    (("layers", 1, "mixer", "decay"), [0.5, 0.5], "decay"),
    (("layers", 1, "mixer", "decay"), [0.5, 0.5, 1.5], "decay"),
    (("layers", 3, "mixer", "heads"), 0, "positive"),
    (("layers", 2, "mlp", "router", "top"), 6, "top"),
    (("layers", 2, "mlp", "kind"), "glu", "not supported"),
    (("norm", "eps"), 0.0, "positive"),
    (("logit_softcap",), -1.0, "positive"),
])
def test_refusals(path, value, words):
    raw = copy.deepcopy(tf.CONFIGS["A"]["config"])
    at = raw
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=words):
        FedipelConfig.from_dict(raw)


def test_missing_keys_are_named():
    raw = copy.deepcopy(tf.CONFIGS["A"]["config"])
    del raw["layers"][0]["mixer"]["diff"]
    with pytest.raises(ConfigError, match=r"layers\[0\].mixer.diff"):
        FedipelConfig.from_dict(raw)


def test_random_weights_load_and_a_wrong_shape_is_refused(tmp_path):
    """Random weights of the architecture load by name; a checkpoint may choose the decay's inner size and nothing else."""
    raw = tf.CONFIGS["A"]["config"]
    folder = write_random_model(raw, 3, tmp_path / "m")
    _, plan = plan_from_config(raw)
    store = WeightStore(folder, Decoder(plan).weight_specs(), plan.ignored_tensors, root="")
    assert store.unexpected == [] and tuple(store.read("l3.mix.w1").shape) == (64, raw["width"])
    decay = torch.exp(-torch.exp(store.read("l3.mix.w0").float()))
    assert 0.3 < float(decay.min()) and float(decay.max()) < 1.0
    store.close()
    w = tf.tensors(raw, 1, rank=9)
    w["l3.mix.u"] = w["l3.mix.u"].t().contiguous()
    bad = tf.write_folder(tmp_path / "bad", raw, w)
    with pytest.raises(WeightError, match="l3.mix.u"):
        WeightStore(bad, Decoder(plan).weight_specs(), plan.ignored_tensors, root="")


# ------------------------------------------------------------------------------------------ pages of a window with kept first positions
@pytest.mark.parametrize("page,window,keep", [(4, 6, 5), (4, 1, 1), (8, 20, 8), (4, 10, 0), (2, 3, 7), (16, 5, 40)])
def test_pages_of_kept_first_positions_stay(page, window, keep):
    """However a request grows, every position that a next token can see has a page, and no page is held beyond those: the pages of the first
    positions stay, the others pass as the window does; a second request in the same pool gets what is free, and all come back."""
    cache = CacheManager([PagedKV(1, 8, window, keep)], page, 64, 2, 256)
    cache.admit("x")
    length = 0
    for n in (1, 2, 9, 1, 1, 30, 1, 3, 17, 1):
        cache.extend("x", length + n)
        table = cache.table(0, "x")
        for at in range(length, length + n):
            for j in range(at + 1):
                if at - j < window or j < keep:
                    assert table[j // page] >= 0, f"position {j}, seen from {at}, has no page"
        length += n
        cache.commit("x", length)
        table = cache.table(0, "x")
        for p in range(-(-length // page)):
            seen = any(length - j < window or j < keep for j in range(p * page, min((p + 1) * page, length)))
            if not seen:
                assert table[p] < 0 or (p + 1) * page > length, f"page {p} is held at length {length} although nothing in it can be seen"
        cache.check()
    assert cache.used_pages()[0] <= -(-keep // page) + -(-window // page) + 1
    missing = cache.pages_missing("x", length + page)[0]
    before = cache.used_pages()[0]
    cache.extend("x", length + page)
    assert cache.used_pages()[0] == before + missing
    cache.admit("y")
    cache.extend("y", 3)
    cache.release("x")
    cache.release("y")
    assert cache.used_pages() == [0]
    cache.check()


# ------------------------------------------------------------------------------------------ the plain pieces by hand
def test_plain_rotation_pairs():
    x = torch.tensor([[[1.0, 0.0, 0.0, 0.0, 9.0]], [[1.0, 0.0, 0.0, 0.0, 9.0]]], dtype=torch.float64)
    a = math.pi / 2
    half = P.rotate(x, torch.tensor([0.0, a], dtype=torch.float64), 4, 1.0, False)
    pair = P.rotate(x, torch.tensor([0.0, a], dtype=torch.float64), 4, 1.0, True)
    assert torch.allclose(half[1, 0], torch.tensor([0.0, 0.0, 1.0, 0.0, 9.0], dtype=torch.float64), atol=1e-12)
    assert torch.allclose(pair[1, 0], torch.tensor([0.0, 1.0, 0.0, 0.0, 9.0], dtype=torch.float64), atol=1e-12)
    assert torch.equal(half[0], x[0]) and torch.equal(pair[0], x[0])


def test_plain_visible_keys():
    seen = P.visible(8, {"size": 3, "keep_first": 2})
    assert seen[7].tolist() == [True, True, False, False, False, True, True, True]
    assert seen[1].tolist() == [True, True] + [False] * 6
    assert P.visible(3, None).int().tolist() == [[1, 0, 0], [1, 1, 0], [1, 1, 1]]


def test_plain_recurrences():
    one = lambda *v: torch.tensor(v, dtype=torch.float64).view(-1, 1, 1)
    o = P.retention_scan(one(1, 1, 2), one(2, 3, 1), one(1, 10, 100), [0.5])
    assert o.flatten().tolist() == [2.0, 31.0, 2 * (0.5 * (0.5 * 2 + 30) + 100)]
    o = P.wkv_scan(one(1, 1, 1), one(2, 3, 1), one(1, 10, 100), one(0.5, 0.25, 0.125), torch.tensor([[7.0]], dtype=torch.float64))
    # the state the second token sees is 2, untouched by its own decay; the third's is 0.25 * 2 + 30
    assert o.flatten().tolist() == [14.0, 2.0 + 210.0, 0.25 * 2 + 30 + 700.0]


def test_plain_router_and_lambda():
    w = {"p.router": torch.eye(3), "p.router.b": torch.tensor([0.0, 0.0, 5.0])}
    idx, wt = P.route(torch.tensor([[1.0, 3.0, -1.0]], dtype=torch.float64), w, "p", 2)
    assert idx.tolist() == [[2, 1]] and torch.allclose(wt, torch.softmax(torch.tensor([[4.0, 3.0]], dtype=torch.float64), -1))
    v = {"p.lq1": torch.tensor([1.0, 2.0]), "p.lk1": torch.tensor([0.5, 0.25]), "p.lq2": torch.tensor([1.0, 0.0]), "p.lk2": torch.tensor([-1.0, 3.0])}
    assert abs(P.diff_lambda(v, "p", 0.8) - (math.e - math.exp(-1.0) + 0.8)) < 1e-12


def test_plain_layer_norm_has_a_bias_and_squared_relu_no_gate():
    w = {"n": torch.tensor([2.0, 1.0]), "n.b": torch.tensor([0.5, -1.0])}
    assert torch.allclose(P.layer_norm(torch.tensor([[3.0, 1.0]], dtype=torch.float64), w, "n", 0.0), torch.tensor([[2.5, -2.0]], dtype=torch.float64))
    w = {"p.up": torch.eye(2), "p.down": torch.eye(2)}
    assert P.relu2_ff(torch.tensor([[3.0, -2.0]], dtype=torch.float64), w, "p").tolist() == [[9.0, 0.0]]


def test_a_state_row_lost_or_a_decay_too_early_would_show():
    """Faults planted in the plain recurrence move its output by far more than the tolerances of the kernels' tests."""
    W, m = 80, {"heads": 3, "dim": 20}
    w = tf.tensors({"vocab": 8, "width": W, "layers": [{"type": "wkv", "mixer": m, "mlp": None}]}, 20, 3)
    h = torch.randn((40, W), generator=torch.Generator().manual_seed(1), dtype=torch.float64)
    want = P.wkv(h, w, "l0.mix", m, 1e-5)
    span = want.abs().max()
    cut = torch.cat([P.wkv(h[:20], w, "l0.mix", m, 1e-5), P.wkv(h[20:], w, "l0.mix", m, 1e-5)])
    assert ((cut - want).abs().amax(1) / span)[20:].median() > 0.05
    no_bonus = dict(w, **{"l0.mix.u": torch.zeros((3, 20))})
    assert ((P.wkv(h, no_bonus, "l0.mix", m, 1e-5) - want).abs().amax(1) / span).median() > 0.05
    still = dict(w, **{f"l0.mix.mu.{s}": torch.zeros(W) for s in "rkvgw"})
    assert ((P.wkv(h, still, "l0.mix", m, 1e-5) - want).abs().amax(1) / span).median() > 0.05
