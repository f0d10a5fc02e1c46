"""Gokosun without a device: the configuration's reader and its refusals, the plan (parts, caches, tensor names and shapes), random weights, and the
plain implementation's own pieces on cases small enough to do by hand; faults planted in the plain form show that the tests' weights reveal them."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_gokosun as P
import tiny_gokosun as tg
from inference_bench_b200.config import ConfigError
from inference_bench_b200.config.gokosun import GokosunConfig
from inference_bench_b200.engine.model import plan_from_config
from inference_bench_b200.parts.base import FixedState, PagedKV, PagedRows, Several
from inference_bench_b200.parts.decoder import Decoder
from inference_bench_b200.weights.loader import WeightError, WeightStore
from inference_bench_b200.weights.random_init import write_random_model

F64 = torch.float64


@pytest.mark.parametrize("name", list(tg.CONFIGS))
def test_config_round_trip_and_plan(name):
    raw = tg.CONFIGS[name]["config"]
    cfg = GokosunConfig.from_dict(raw)
    assert GokosunConfig.from_dict(cfg.to_dict()) == cfg
    _, plan = plan_from_config(raw)
    dec = Decoder(plan)
    specs = {s.name: s for s in dec.weight_specs()}
    made = tg.tensors(raw, 1)
    assert set(specs) == set(made) and all(specs[n].fits(tuple(made[n].shape)) for n in made)
    assert [e.layer for e in plan.schedule] == list(range(len(raw["layers"])))
    for l, need in zip(raw["layers"], dec.cache_needs()):
        m = l["mixer"]
        if l["type"] == "mlstm":
            assert need == Several((FixedState((m["heads"], m["dim"], m["vdim"] + 1), torch.float32), FixedState((m["heads"],), torch.float32)))
        elif l["type"] == "latent_attention":
            assert need == PagedRows(m["kv_rank"] + m["rot_dim"], None)
        else:
            row = max(m["dim"], m["vdim"])
            assert need == PagedKV(m["kv_heads"], row + row % 2, None)


def test_which_layer_gives_the_values_that_others_mix_with():
    cfg = GokosunConfig.from_dict(tg.CONFIGS["A"]["config"])
    assert cfg.first_mixed == 3
    _, plan = plan_from_config(tg.CONFIGS["A"]["config"])
    assert [l.mixer.params.get("value_mix") for l in plan.layers] == [None, None, None, "first", None, "mix", None]
    raw = copy.deepcopy(tg.CONFIGS["A"]["config"])
    raw["layers"][1]["mixer"]["v_mix"] = True
    raw["layers"][1]["mixer"]["vdim"] = 20
    assert GokosunConfig.from_dict(raw).first_mixed == 1
    del raw["layers"][5]["mixer"]["v_mix"]
    assert [l.mixer.params.get("value_mix") for l in plan_from_config(raw)[1].layers] == [None, "first", None, "mix", None, None, None]


@pytest.mark.parametrize("path,value,words", [
    (("layers", 0, "type"), "mamba2", "not supported"),
    (("layers", 1, "mixer", "kv_heads"), 3, "multiple"),
    (("layers", 1, "mixer", "rot", "dims"), 7, "even"),
    (("layers", 1, "mixer", "rot", "dims"), 18, "at most 16"),
    (("layers", 0, "mixer", "rot", "dims"), 10, "at most 8"),
    (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0, "positive"),
    (("layers", 0, "mixer", "q_rank"), 0, "positive"),
    (("layers", 1, "mixer", "dim"), 258, "at most 256"),
    (("layers", 2, "mixer", "dim"), 513, "above 512"),
    (("layers", 2, "mixer", "gate_cap"), -1.0, "positive"),
    (("layers", 5, "mixer", "vdim"), 21, "mixes its values"),
    (("layers", 0, "mlp", "router", "top"), 6, "top"),
    (("layers", 0, "mlp", "expert", "limit"), 0.0, "positive"),
    (("layers", 0, "mlp", "shared", "limit"), -2.0, "positive"),
    (("layers", 3, "mlp", "limit"), 0.0, "positive"),
    (("layers", 3, "mlp", "kind"), "glu", "not supported"),
    (("norm", "eps"), 0.0, "positive"),
    (("layers",), [], "non-empty"),
])
def test_refusals(path, value, words):
    raw = copy.deepcopy(tg.CONFIGS["A"]["config"])
    at = raw
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=words):
        GokosunConfig.from_dict(raw)


@pytest.mark.parametrize("layer,key", [(0, "q_rank"), (0, "scale"), (2, "gate_cap"), (1, "vdim")])
def test_missing_keys_are_named(layer, key):
    raw = copy.deepcopy(tg.CONFIGS["A"]["config"])
    del raw["layers"][layer]["mixer"][key]
    with pytest.raises(ConfigError, match=rf"layers\[{layer}\].mixer.{key}"):
        GokosunConfig.from_dict(raw)


def test_random_weights_load_and_a_wrong_shape_is_refused(tmp_path):
    raw = tg.CONFIGS["A"]["config"]
    folder = write_random_model(raw, 3, tmp_path / "m")
    _, plan = plan_from_config(raw)
    store = WeightStore(folder, Decoder(plan).weight_specs(), plan.ignored_tensors, root="")
    assert store.unexpected == []
    assert 0.8 < float(torch.sigmoid(store.read("l2.mix.f.b").float()).min()) and tuple(store.read("l5.mix.vmix").shape) == ()
    store.close()
    w = tg.tensors(raw, 1)
    w["l3.mix.vmix"] = torch.tensor(0.5, dtype=torch.bfloat16)     # a checkpoint may carry the first layer's, which is not used
    WeightStore(tg.write_folder(tmp_path / "more", raw, w), Decoder(plan).weight_specs(), plan.ignored_tensors, root="").close()
    w["l1.mix.q.norm"] = w["l1.mix.q.norm"][:16].contiguous()      # a norm over one head instead of all
    with pytest.raises(WeightError, match="l1.mix.q.norm"):
        WeightStore(tg.write_folder(tmp_path / "bad", raw, w), Decoder(plan).weight_specs(), plan.ignored_tensors, root="")


# ------------------------------------------------------------------------------------------ the plain pieces by hand
def test_plain_rotation_pairs_and_rescaled_frequencies():
    x = torch.tensor([[[1.0, 0.0, 0.0, 0.0, 9.0]], [[1.0, 0.0, 0.0, 0.0, 9.0]]], dtype=F64)
    pos, rot = torch.tensor([0.0, math.pi / 2], dtype=F64), {"dims": 4, "base": 1.0}
    assert torch.allclose(P.rotate(x, pos, rot, False)[1, 0], torch.tensor([0.0, 0.0, 1.0, 0.0, 9.0], dtype=F64), atol=1e-12)
    assert torch.allclose(P.rotate(x, pos, rot, True)[1, 0], torch.tensor([0.0, 1.0, 0.0, 0.0, 9.0], dtype=F64), atol=1e-12)
    # dims 8, base 16: frequencies 1, 1/2, 1/4, 1/8; a pair turns `original` f / (2 pi) times: with original = 8 pi, 4, 2, 1 and 1/2 times.
    # fast 2 (pair 1), slow 1/2 (pair 3): pairs 0, 1 keep theirs, pair 2 has the mean of both, pair 3 a quarter
    f, amp = P.yarn_frequencies(8, 16.0, {"factor": 4.0, "original": 8 * math.pi, "fast": 2.0, "slow": 0.5})
    assert torch.allclose(f, torch.tensor([1.0, 0.5, 0.25 * (0.5 + 0.125), 0.125 / 4], dtype=F64), atol=1e-12) and abs(amp - 1.0 - 0.1 * math.log(4.0)) < 1e-12
    # the ramp's ends are cut to the range: everything is slow where even pair 0 turns less than `fast` and `slow` times
    f, _ = P.yarn_frequencies(4, 16.0, {"factor": 2.0, "original": 1.0, "fast": 64.0, "slow": 32.0})
    assert torch.allclose(f, torch.tensor([1.0, 0.125], dtype=F64))     # lo = 0, hi = max(hi - lo, 0.001) past pair 0


def test_plain_memory_scan():
    one = lambda *v: torch.tensor(v, dtype=F64).view(-1, 1, 1)
    col = lambda *v: torch.tensor(v, dtype=F64).view(-1, 1)
    # i = f = 0: m stays 0, S = sum k v, n = sum k; with q = 1: 2 / 2, (2 + 30) / 5
    o = P.memory_scan(one(1, 1), one(2, 3), one(1, 10), col(0, 0), col(0, 0))
    assert torch.allclose(o.flatten(), torch.tensor([2.0 / (2.0 + 1e-6), 32.0 / (5.0 + 1e-6)], dtype=F64))
    # an input gate of ln 4: m becomes ln 4, the old state counts a quarter, the bound is 1/4 (|n q| = 0.25 * 2 + 3); small keys meet the bound
    o = P.memory_scan(one(1, 1), one(2, 3), one(1, 10), col(0, math.log(4.0)), col(0, 0))
    assert abs(o[1].item() - (0.25 * 2 + 30) / (3.5 + 1e-6)) < 1e-12
    o = P.memory_scan(one(1), one(0.01), one(5), col(0), col(0))
    assert abs(o[0].item() - 0.05 / (1.0 + 1e-6)) < 1e-12
    # a very negative input gate: m follows the forget gate down, the bound e^(-m) grows
    o = P.memory_scan(one(1), one(2), one(1), col(-9.0), col(-1.0))
    assert abs(o[0].item() - 2 * math.exp(-8.0) / (math.exp(1.0) + 1e-6)) < 1e-12


def test_plain_sink_counts_once_and_has_no_value():
    p = P.causal_softmax(torch.zeros((3, 3), dtype=F64), math.log(2.0))
    assert torch.allclose(p.sum(-1), torch.tensor([1 / 3, 2 / 4, 3 / 5], dtype=F64)) and p[0, 1] == 0 and p[1, 2] == 0


def test_plain_clamped_pair_and_router():
    g = torch.tensor([5.0, -3.0, 1.0], dtype=F64)
    u = torch.tensor([0.5, 9.0, -9.0], dtype=F64)
    want = [2 / (1 + math.exp(-1.702 * 2)) * 1.5, -3 / (1 + math.exp(1.702 * 3)) * 3.0, 1 / (1 + math.exp(-1.702)) * -1.0]
    assert torch.allclose(P.clamped_glu(g, u, 2.0), torch.tensor(want, dtype=F64))
    w = {"p.router": torch.eye(3), "p.correction": torch.tensor([0.0, -1.0, 0.9])}
    idx, wt = P.route(torch.tensor([[1.0, 3.0, -1.0]], dtype=F64), w, "p", 2, 2.0)
    s = torch.sigmoid(torch.tensor([-1.0, 1.0], dtype=F64))
    assert idx.tolist() == [[2, 0]] and torch.allclose(wt, (2.0 * s / s.sum())[None])


def test_plain_layer_norm_has_a_bias():
    w = {"n": torch.tensor([2.0, 1.0]), "n.b": torch.tensor([0.5, -1.0])}
    assert torch.allclose(P.layer_norm(torch.tensor([[3.0, 1.0]], dtype=F64), w, "n", 0.0), torch.tensor([[2.5, -2.0]], dtype=F64))


# ------------------------------------------------------------------------------------------ faults that the tests' weights show
def _moved(name, change):
    """By how much a changed configuration or changed weights move the logits' rows, of the largest logit."""
    raw = copy.deepcopy(tg.CONFIGS[name]["config"])
    w = tg.tensors(raw, tg.CONFIGS[name]["seed"])
    toks = list(range(3, 63))
    want = P.logits(raw, w, toks)
    change(raw, w)
    return (P.logits(raw, w, toks) - want).abs().amax(1) / want.abs().max()


@pytest.mark.parametrize("what,change", [
    ("no sink", lambda c, w: w["l0.mix.sink"].fill_(-30.0)),
    ("no rescaling", lambda c, w: c["layers"][0]["mixer"]["rot"].pop("scaling")),
    ("no value mixing", lambda c, w: w["l5.mix.vmix"].zero_()),
    ("mixing with another layer's values", lambda c, w: w["l5.mix.vmix"].fill_(1.0)),
    ("another gate cap", lambda c, w: c["layers"][2]["mixer"].update(gate_cap=50.0)),
    ("one limit for all experts", lambda c, w: c["layers"][0]["mlp"]["shared"].update(limit=1.5)),
    ("no correction", lambda c, w: w["l0.mlp.correction"].zero_()),
    ("no norm bias", lambda c, w: w["l3.norm1.b"].zero_()),
])
def test_a_lost_mechanism_would_show(what, change):
    assert _moved("A", change).median().item() > 3e-3, what


def test_a_state_lost_between_portions_or_a_maximum_that_starts_elsewhere_would_show():
    W, m = 80, {"heads": 3, "dim": 20, "vdim": 12, "gate_cap": 5.0}
    w = tg.tensors({"vocab": 8, "width": W, "layers": [{"type": "mlstm", "mixer": m, "mlp": None}]}, 20)
    h = torch.randn((40, W), generator=torch.Generator().manual_seed(1), dtype=F64)
    want = P.memory(h, w, "l0.mix", m, 1e-5)
    cut = torch.cat([P.memory(h[:20], w, "l0.mix", m, 1e-5), P.memory(h[20:], w, "l0.mix", m, 1e-5)])
    assert ((cut - want).abs().amax(1) / want.abs().max())[20:].median() > 0.03
    # the bound e^(-m) with m from minus infinity would be the first input gate's own: the scan's first row tells them apart
    q = k = torch.full((1, 1, 1), 0.1, dtype=F64)
    low = P.memory_scan(q, k, k * 10, torch.full((1, 1), -2.0, dtype=F64), torch.full((1, 1), -0.1, dtype=F64))
    assert abs(low.item() - 0.1 * math.exp(-1.9) * 0.1 / math.exp(0.1)) < 1e-6
