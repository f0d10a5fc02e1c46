"""Tiny Fedipel configurations for the tests, with weights the tests make themselves. They differ in every size and constant: width (a
multiple of 8 or not), the order of the three mixers, query and key/value head counts (equal, grouped by two, by eight), maps of a head that
are partly, wholly or not turned, value heads of another size than two maps, windows shorter than a page, of several pages, of one position
or none, kept first positions fewer than a page, more than a page, more than the window, or none; layers that read an earlier layer's keys
with a wider or a narrower mask; decays of 0 and 1 among the heads; decay ranks of 1 to 24; dense, routed (one expert, one choice, all
experts chosen) and absent feed-forwards, with and without a shared expert of the experts' size or another; residual multipliers and logit
caps of their own or none; norm epsilon, page size."""
from __future__ import annotations

import json
from pathlib import Path

import torch


def _att(heads, kv_heads, dim, vdim, window, keep, dims, base, scale, diff, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, "rot": {"base": base, "dims": dims},
         "mask": None if window is None else {"size": window, "keep_first": keep}}
    return m if kv_from is None else dict(m, kv_from=kv_from)


def _ret(heads, dim, vdim, decay, dims, base):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": {"base": base, "dims": dims}}


def _moe(ff, experts, top, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return f if shared is None else dict(f, shared={"ff": shared})


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


CONFIGS = {
    # attention first, read by a later layer whose window is wider and by one that keeps more; heads no tensor-core kernel takes; a layer
    # without a feed-forward after each kind of mixer but the last
    "A": dict(seed=61, page_size=16, rank=3, config={
        "architecture": "Fedipel", "vocab": 300, "width": 80, "norm": {"eps": 1e-5}, "residual_mult": 0.6, "logit_softcap": 20.0,
        "layers": [_layer("attention", _att(4, 2, 16, 24, 9, 3, 8, 1000.0, 0.4, 0.4), _dense(40)),
                   _layer("retention", _ret(3, 20, 12, (0.5, 0.9, 0.99), 12, 300.0), None),
                   _layer("attention", _att(2, 2, 16, 24, 40, 1, 8, 1000.0, 0.3, 0.7, kv_from=0), _moe(24, 5, 2, 56)),
                   _layer("wkv", {"heads": 3, "dim": 20}, None),
                   _layer("attention", _att(6, 2, 16, 24, 5, 19, 8, 1000.0, 0.5, 0.2, kv_from=0), None),
                   _layer("wkv", {"heads": 2, "dim": 36}, _moe(16, 4, 4))]}),
    # a width that is no multiple of 8; a recurrence first; attention without a window, nothing turned, as many kv heads as heads; decays of 1
    # and 0; no cap on the logits, no residual multiplier; a decay of rank 1; one expert of one; one choice of three
    "B": dict(seed=62, page_size=8, rank=1, config={
        "architecture": "Fedipel", "vocab": 257, "width": 132, "norm": {"eps": 1e-6}, "residual_mult": 1.0, "logit_softcap": None,
        "layers": [_layer("wkv", {"heads": 5, "dim": 24}, _moe(36, 1, 1, 20)),
                   _layer("retention", _ret(4, 12, 40, (1.0, 0.0, 0.8, 0.999), 12, 50.0), _moe(28, 3, 1)),
                   _layer("attention", _att(3, 3, 10, 14, None, 0, 0, 10.0, 0.5, 0.5), _dense(100)),
                   _layer("retention", _ret(2, 34, 6, (0.97, 0.3), 0, 10.0), None)]}),
    # heads of 64 and 128 (two maps and values alike), eight query heads on one kv head, windows of three pages and of 70 with more than a page
    # kept, a reader with a narrower window; sizes the tensor-core products take everywhere
    "C": dict(seed=63, page_size=16, rank=24, config={
        "architecture": "Fedipel", "vocab": 512, "width": 192, "norm": {"eps": 1e-5}, "residual_mult": 0.4, "logit_softcap": 12.0,
        "layers": [_layer("attention", _att(8, 1, 32, 64, 48, 5, 32, 10000.0, 0.25, 0.3), _moe(64, 8, 3, 128)),
                   _layer("wkv", {"heads": 3, "dim": 64}, _dense(128)),
                   _layer("attention", _att(3, 3, 64, 128, 70, 20, 16, 500000.0, 0.15, 0.6), _moe(128, 6, 2, 64)),
                   _layer("retention", _ret(2, 64, 128, (0.98, 0.6), 32, 10000.0), _moe(64, 16, 4)),
                   _layer("attention", _att(6, 3, 64, 128, 33, 2, 16, 500000.0, 0.1, 0.45, kv_from=2), _dense(96))]}),
    # one layer, a window of one position beside more kept positions than that
    "D": dict(seed=64, page_size=32, rank=2, config={
        "architecture": "Fedipel", "vocab": 100, "width": 48, "norm": {"eps": 1e-6}, "residual_mult": 1.7, "logit_softcap": 5.0,
        "layers": [_layer("attention", _att(2, 1, 12, 8, 1, 6, 4, 100.0, 0.6, 0.35), _dense(24))]}),
}


def tensors(config: dict, seed: int, rank: int = 4) -> dict[str, torch.Tensor]:
    """Random bfloat16 tensors: matrices N(0, gain / sqrt(fan-in)) so that activations stay of order one, norm weights around one, norm biases
    N(0, 0.2), mixing weights in (0, 1), the bonus N(0, 0.7), decay offsets in (-5, 0), biases N(0, 0.3)."""
    g = torch.Generator().manual_seed(seed)
    W, out = config["width"], {}

    def mat(name, n, k, gain=1.0):
        out[name] = (torch.randn((n, k), generator=g) * gain / k ** 0.5).to(torch.bfloat16)

    def noise(name, shape, std, centre=0.0):
        out[name] = (centre + torch.randn(shape, generator=g) * std).to(torch.bfloat16)

    def norm(name):
        noise(name, (W,), 0.2, 1.0), noise(f"{name}.b", (W,), 0.2)

    out["embed"] = torch.randn((config["vocab"], W), generator=g).to(torch.bfloat16)
    norm("embed.norm")
    for i, l in enumerate(config["layers"]):
        m, p = l["mixer"], f"l{i}.mix"
        norm(f"l{i}.norm1")
        H, D = m["heads"], m["dim"]
        if l["type"] == "retention":
            V = m["vdim"]
            mat(f"{p}.q", H * D, W), mat(f"{p}.k", H * D, W), mat(f"{p}.v", H * V, W), mat(f"{p}.g", H * V, W, 2.0), mat(f"{p}.o", W, H * V, 1.5)
        elif l["type"] == "wkv":
            C = H * D
            for s in "rkvgw":
                out[f"{p}.mu.{s}"] = torch.rand((W,), generator=g).to(torch.bfloat16)
            for s in "rkv":
                mat(f"{p}.{s}", C, W)
            mat(f"{p}.g", C, W, 2.0), mat(f"{p}.w1", rank, W, 1.5), mat(f"{p}.w2", C, rank, 1.5)
            out[f"{p}.w0"] = (torch.rand((C,), generator=g) * 5.0 - 5.0).to(torch.bfloat16)
            noise(f"{p}.u", (H, D), 0.7), noise(f"{p}.norm", (C,), 0.2, 1.0), mat(f"{p}.o", W, C, 1.5)
        else:
            G, V = m["kv_heads"], m["vdim"]
            mat(f"{p}.q", H * 2 * D, W, 2.0), noise(f"{p}.q.b", (H * 2 * D,), 0.3)
            if m.get("kv_from") is None:
                mat(f"{p}.k", G * 2 * D, W, 2.0), noise(f"{p}.k.b", (G * 2 * D,), 0.3), mat(f"{p}.v", G * V, W), noise(f"{p}.v.b", (G * V,), 0.3)
            for s in ("lq1", "lk1", "lq2", "lk2"):
                noise(f"{p}.{s}", (D,), 0.3)
            mat(f"{p}.o", W, H * V, 1.5)
        f, q = l.get("mlp"), f"l{i}.mlp"
        if f is None:
            continue
        norm(f"l{i}.norm2")
        if f["kind"] == "dense":
            mat(f"{q}.gate", f["ff"], W, 1.5), mat(f"{q}.up", f["ff"], W), mat(f"{q}.down", W, f["ff"], 1.5)
            continue
        E, F = f["router"]["experts"], f["expert"]["ff"]
        mat(f"{q}.router", E, W, 2.0), noise(f"{q}.router.b", (E,), 0.3)
        for e in range(E):
            mat(f"{q}.e{e}.up", F, W, 1.5), mat(f"{q}.e{e}.down", W, F)
        if f.get("shared"):
            S = f["shared"]["ff"]
            mat(f"{q}.shared.up", S, W, 1.5), mat(f"{q}.shared.down", W, S), mat(f"{q}.shared.sg", 1, W)
    norm("final.norm")
    mat("head", config["vocab"], W, 2.0)
    return out


def write_folder(out_dir, config: dict, weights: dict) -> Path:
    from inference_bench_b200.weights.safetensors_io import write_safetensors
    out = Path(out_dir)
    out.mkdir(parents=True, exist_ok=True)
    (out / "config.json").write_text(json.dumps(config, indent=1))
    write_safetensors(out / "model.safetensors", weights, {"format": "pt"})
    return out


def write_model(name: str, out_dir) -> Path:
    c = CONFIGS[name]
    return write_folder(out_dir, c["config"], tensors(c["config"], c["seed"], c["rank"]))
