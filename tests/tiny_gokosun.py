"""Tiny Gokosun configurations for the tests, with weights the tests make themselves. They differ in every size and constant: width (a
multiple of 8 or not), the order of the three mixers, memory heads whose values are smaller than, as large as and larger than their keys, gate
caps, query and key/value head counts (equal, grouped by two, by eight, one), heads partly, wholly or not turned, value heads of another size
than keys, layers with and without mixed values (the first of them first, last or alone), latent ranks the tensor-core kernels take and do
not, query latents of a few values and of more than the width, rotations with and without rescaling (a ramp inside, before and beyond the pairs),
dense, routed (one expert, one choice, all chosen) and absent feed-forwards, shared experts of the experts' size, of a multiple, of another size
or none, limits and route scales of their own; norm epsilon, page size."""
from __future__ import annotations

import json
from pathlib import Path

import torch


def _att(heads, kv_heads, dim, vdim, dims, base, scale, v_mix=True):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix, "rot": {"base": base, "dims": dims}}


def _mem(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def _lat(heads, dim, rot, vdim, kv_rank, q_rank, base, scale, yarn=None):
    r = {"base": base, "dims": rot}
    if yarn:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale, "rot": r}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(ff, limit, experts, top, scale, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "scale": scale}}
    return f if shared is None else dict(f, shared={"ff": shared[0], "limit": shared[1]})


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


CONFIGS = {
    # a latent layer first; the first layer with mixed values after one without; a layer without a feed-forward after each kind of mixer
    "A": dict(seed=71, page_size=16, config={
        "architecture": "Gokosun", "vocab": 300, "width": 80, "norm": {"eps": 1e-5},
        "layers": [_layer("latent_attention", _lat(3, 12, 8, 20, 24, 40, 1000.0, 0.3, (4.0, 64, 8.0, 1.0)), _moe(24, 1.5, 5, 2, 1.5, (48, 0.8))),
                   _layer("attention", _att(4, 2, 16, 24, 8, 500.0, 0.4, v_mix=False), None),
                   _layer("mlstm", _mem(3, 20, 12, 5.0), None),
                   _layer("attention", _att(4, 4, 20, 10, 20, 1000.0, 0.3), _dense(40, 1.2)),
                   _layer("latent_attention", _lat(2, 6, 4, 10, 18, 5, 50.0, 0.5), None),
                   _layer("attention", _att(6, 2, 12, 20, 4, 100.0, 0.35), _moe(16, 0.7, 4, 4, 0.5)),
                   _layer("mlstm", _mem(2, 9, 36, 15.0), _dense(56, 3.0))]}),
    # a width that is no multiple of 8; the memory first; one layer with values to mix, alone; a shared expert of another size than the experts'
    "B": dict(seed=72, page_size=8, config={
        "architecture": "Gokosun", "vocab": 257, "width": 132, "norm": {"eps": 1e-6},
        "layers": [_layer("mlstm", _mem(5, 24, 24, 8.0), _moe(36, 2.0, 1, 1, 3.0, (20, 1.0))),
                   _layer("attention", _att(3, 3, 10, 14, 0, 10.0, 0.5), _moe(28, 1.0, 3, 1, 1.0)),
                   _layer("latent_attention", _lat(5, 10, 6, 7, 33, 150, 300.0, 0.25, (16.0, 32, 2.0, 0.25)), _dense(100, 2.5)),
                   _layer("mlstm", _mem(1, 34, 6, 3.0), None)]}),
    # heads of 64 and 128, sizes the tensor-core kernels and products take everywhere, shared experts of one and two of the experts' sizes
    "C": dict(seed=73, page_size=16, config={
        "architecture": "Gokosun", "vocab": 512, "width": 256, "norm": {"eps": 1e-5},
        "layers": [_layer("attention", _att(8, 1, 64, 64, 64, 10000.0, 0.125), _moe(64, 1.0, 8, 3, 2.5, (128, 2.0))),
                   _layer("mlstm", _mem(3, 64, 96, 15.0), _dense(192, 2.0)),
                   _layer("latent_attention", _lat(6, 32, 16, 48, 64, 96, 5000.0, 0.18, (2.0, 128, 16.0, 1.0)), _moe(128, 2.0, 6, 2, 1.0, (128, 1.0))),
                   _layer("attention", _att(2, 1, 128, 64, 32, 500000.0, 0.1), _dense(96, 1.5)),
                   _layer("mlstm", _mem(2, 128, 64, 10.0), _moe(64, 1.2, 16, 4, 1.7, (64, 1.6)))]}),
    # one layer of one head
    "D": dict(seed=74, page_size=32, config={
        "architecture": "Gokosun", "vocab": 100, "width": 48, "norm": {"eps": 1e-6},
        "layers": [_layer("mlstm", _mem(1, 12, 8, 2.0), _dense(24, 0.9))]}),
}


def tensors(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """Random bfloat16 tensors: matrices N(0, gain / sqrt(fan-in)) so that activations stay of order one, norm weights around one, norm biases
    N(0, 0.2), forget gates' biases in (-1, 6), input gates' N(0, 1), sinks in (0, 4), corrections N(0, 0.3), mixing numbers in (0.2, 0.8)."""
    g = torch.Generator().manual_seed(seed)
    W, out = config["width"], {}
    first = next((i for i, l in enumerate(config["layers"]) if l["mixer"].get("v_mix")), None)

    def mat(name, n, k, gain=1.0):
        out[name] = (torch.randn((n, k), generator=g) * gain / k ** 0.5).to(torch.bfloat16)

    def noise(name, shape, std, centre=0.0):
        out[name] = (centre + torch.randn(shape, generator=g) * std).to(torch.bfloat16)

    def between(name, shape, lo, hi):
        out[name] = (lo + torch.rand(shape, generator=g) * (hi - lo)).to(torch.bfloat16)

    def gated(name, ff):
        mat(f"{name}.gate", ff, W, 1.5), mat(f"{name}.up", ff, W, 1.5), mat(f"{name}.down", W, ff)

    out["embed"] = torch.randn((config["vocab"], W), generator=g).to(torch.bfloat16)
    for i, l in enumerate(config["layers"]):
        m, p = l["mixer"], f"l{i}.mix"
        noise(f"l{i}.norm1", (W,), 0.2, 1.0), noise(f"l{i}.norm1.b", (W,), 0.2)
        H, D, V = m["heads"], m["dim"], m["vdim"]
        if l["type"] == "mlstm":
            mat(f"{p}.q", H * D, W), mat(f"{p}.k", H * D, W), mat(f"{p}.v", H * V, W), mat(f"{p}.g", H * V, W, 2.0), mat(f"{p}.o", W, H * V, 2.0)
            mat(f"{p}.i", H, W, 2.0), noise(f"{p}.i.b", (H,), 1.0), mat(f"{p}.f", H, W, 1.0), between(f"{p}.f.b", (H,), -1.0, 6.0), noise(f"{p}.norm", (H * V,), 0.2, 1.0)
        elif l["type"] == "latent_attention":
            R, K, Q = m["rot_dim"], m["kv_rank"], m["q_rank"]
            mat(f"{p}.dq", Q, W), noise(f"{p}.dq.norm", (Q,), 0.2, 1.0), mat(f"{p}.uq", H * (D + R), Q, 2.0)
            mat(f"{p}.dkv", K + R, W), noise(f"{p}.dkv.norm", (K,), 0.2, 1.0), mat(f"{p}.uk", H * D, K, 1.5), mat(f"{p}.uv", H * V, K)
            between(f"{p}.sink", (H,), 0.0, 4.0), mat(f"{p}.o", W, H * V, 2.0)
        else:
            G = m["kv_heads"]
            mat(f"{p}.q", H * D, W), mat(f"{p}.k", G * D, W), mat(f"{p}.v", G * V, W), mat(f"{p}.o", W, H * V, 2.0)
            noise(f"{p}.q.norm", (H * D,), 0.3, 1.5), noise(f"{p}.k.norm", (G * D,), 0.3, 1.5)
            if m["v_mix"] and i != first:
                between(f"{p}.vmix", (), 0.2, 0.8)
        f, q = l.get("mlp"), f"l{i}.mlp"
        if f is None:
            continue
        if f["kind"] == "dense":
            gated(q, f["ff"])
            continue
        mat(f"{q}.router", f["router"]["experts"], W, 2.0), noise(f"{q}.correction", (f["router"]["experts"],), 0.3)
        for e in range(f["router"]["experts"]):
            gated(f"{q}.e{e}", f["expert"]["ff"])
        if f.get("shared"):
            gated(f"{q}.shared", f["shared"]["ff"])
    noise("final.norm", (W,), 0.2, 1.0), noise("final.norm.b", (W,), 0.2)
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
    return write_folder(out_dir, c["config"], tensors(c["config"], c["seed"]))
