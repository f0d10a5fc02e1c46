"""A plain, slow Fedipel: one function per mechanism, written from the architecture's equations in double precision with torch
on the CPU. It shares no code with the engine and is what the engine's kernels are compared with.

Notation: x [T, W] is one sequence's residual stream (rows are positions 0..T-1), `cfg` the dictionary of config.json, `w` a
dictionary name -> tensor (any floating dtype; everything is widened to float64).

    x = LN(embed[tokens]);   per layer  x = x + m mixer(LN1(x));  x = x + m ff(LN2(x))   (a layer may have no feed-forward)
    logits = c tanh(head LN(x) / c)
LN is a layer norm with a weight and a bias; mixers are retention, a recurrence with a data-dependent decay per channel behind a token
shift, or differential attention over a window and the first tokens; feed-forwards are SiLU-gated or experts with squared ReLUs.
"""
from __future__ import annotations

import contextlib
import math

import torch

F64 = torch.float64


ROUND = False     # True (`rounded`): what a bfloat16 engine stores in 16 bits is rounded: the inputs of every matrix product, turned queries and keys, values,
                  # attention outputs. How far that moves a row says how far an engine's own rounding may.


def d(t):
    return t.to(F64)


def rnd(t):
    return t.to(torch.bfloat16).to(F64) if ROUND else t


def lin(h, w):
    """h w^T for a stored matrix [out, in]."""
    return rnd(h) @ d(w).T


@contextlib.contextmanager
def rounded():
    global ROUND
    ROUND = True
    try:
        yield
    finally:
        ROUND = False


# ------------------------------------------------------------------------------------------ small pieces
def layer_norm(x, w, name, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * d(w[name]) + d(w[f"{name}.b"])


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def relu2(z):
    return torch.clamp(z, min=0) ** 2


def rotate(x, positions, dims, base, interleaved):
    """x [T, heads, dim]: the first `dims` entries are turned in pairs by the angles position * base^(-2i/dims); pair i is (i, i + dims/2), or
    (2i, 2i + 1) when interleaved."""
    n = dims // 2
    if n == 0:
        return x
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(n)], dtype=F64)
    a = d(positions)[:, None, None] * f
    cos, sin = torch.cos(a), torch.sin(a)
    if interleaved:
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        turned = torch.stack([u * cos - v * sin, v * cos + u * sin], -1).flatten(-2)
    else:
        u, v = x[..., :n], x[..., n:dims]
        turned = torch.cat([u * cos - v * sin, v * cos + u * sin], -1)
    return torch.cat([turned, x[..., dims:]], -1)


# ------------------------------------------------------------------------------------------ retention
def retention_scan(q, k, v, decay):
    """q, k [T, H, D], v [T, H, V]: S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    T, H, D = q.shape
    g = torch.tensor(decay, dtype=F64)[:, None, None]
    S = torch.zeros((H, D, v.shape[2]), dtype=F64)
    o = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for t in range(T):
        S = g * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o


def retention(h, w, p, m, eps):
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    dims, base = int(m["rot"]["dims"]), float(m["rot"]["base"])
    pos = torch.arange(T)
    q = rotate(lin(h, w[f"{p}.q"]).view(T, H, D), pos, dims, base, False)
    k = rotate(lin(h, w[f"{p}.k"]).view(T, H, D), pos, dims, base, False) / math.sqrt(D)
    v = lin(h, w[f"{p}.v"]).view(T, H, V)
    o = rms_unit(retention_scan(q, k, v, [float(x) for x in m["decay"]]), eps).reshape(T, H * V)
    return lin(o * silu(lin(h, w[f"{p}.g"])), w[f"{p}.o"])


# ------------------------------------------------------------------------------------------ the recurrence with a decay per channel
def wkv_scan(r, k, v, decay, u):
    """r, k, decay [T, H, D], v [T, H, D], u [H, D]: o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t, then S_t = diag(decay_t) S_(t-1) + k_t v_t^T."""
    T, H, D = r.shape
    S = torch.zeros((H, D, v.shape[2]), dtype=F64)
    o = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = ((S + u[:, :, None] * kv) * r[t][:, :, None]).sum(1)
        S = decay[t][:, :, None] * S + kv
    return o


def wkv(h, w, p, m, eps):
    T = h.shape[0]
    H, D = int(m["heads"]), int(m["dim"])
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], 0)
    mix = {s: h + (before - h) * d(w[f"{p}.mu.{s}"]) for s in "rkvgw"}
    r, k, v = (lin(mix[s], w[f"{p}.{s}"]).view(T, H, D) for s in "rkv")
    gate = silu(lin(mix["g"], w[f"{p}.g"]))
    z = torch.tanh(lin(mix["w"], w[f"{p}.w1"])) @ d(w[f"{p}.w2"]).T + d(w[f"{p}.w0"])
    o = wkv_scan(r, k, v, torch.exp(-torch.exp(z)).view(T, H, D), d(w[f"{p}.u"]).view(H, D))
    return lin(rms_unit(o, eps).reshape(T, H * D) * d(w[f"{p}.norm"]) * gate, w[f"{p}.o"])


# ------------------------------------------------------------------------------------------ differential attention
def visible(T, mask):
    """[T, T]: position i sees j <= i that lies within the last `size` positions or among the first `keep_first`."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    if not mask:
        return j <= i
    return (j <= i) & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first") or 0)))


def masked_attention(q, k, v, seen, scale):
    """One map: q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V], an ordinary softmax over the visible keys."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for a in range(H):
        b = a // (H // G)
        out[:, a] = torch.softmax(((q[:, a] @ k[:, b].T) * scale).masked_fill(~seen, -math.inf), -1) @ v[:, b]
    return out


def diff_lambda(w, p, diff):
    return math.exp(float((d(w[f"{p}.lq1"]) * d(w[f"{p}.lk1"])).sum())) - math.exp(float((d(w[f"{p}.lq2"]) * d(w[f"{p}.lk2"])).sum())) + diff


def attention_kv(h, w, p, m):
    """The keys of both maps, turned, [T, G, 2, D], and the values [T, G, V]."""
    T = h.shape[0]
    G, D, V = int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    k = (lin(h, w[f"{p}.k"]) + d(w[f"{p}.k.b"])).view(T, G * 2, D)
    k = rotate(k, torch.arange(T), int(m["rot"]["dims"]), float(m["rot"]["base"]), True).view(T, G, 2, D)
    return rnd(k), rnd(lin(h, w[f"{p}.v"]) + d(w[f"{p}.v.b"])).view(T, G, V)


def diff_attention(h, w, p, m, eps, kv):
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    k, v = kv
    q = (lin(h, w[f"{p}.q"]) + d(w[f"{p}.q.b"])).view(T, H * 2, D)
    q = rnd(rotate(q, torch.arange(T), int(m["rot"]["dims"]), float(m["rot"]["base"]), True)).view(T, H, 2, D)
    seen, scale, diff = visible(T, m["mask"]), float(m["scale"]), float(m["diff"])
    a1, a2 = (rnd(masked_attention(q[:, :, i], k[:, :, i], v, seen, scale)) for i in (0, 1))
    o = rms_unit(a1 - diff_lambda(w, p, diff) * a2, eps) * (1.0 - diff)
    return lin(o.reshape(T, H * V), w[f"{p}.o"])


# ------------------------------------------------------------------------------------------ feed-forwards
def dense_ff(h, w, p):
    return lin(silu(lin(h, w[f"{p}.gate"])) * lin(h, w[f"{p}.up"]), w[f"{p}.down"])


def relu2_ff(h, w, p):
    return lin(relu2(lin(h, w[f"{p}.up"])), w[f"{p}.down"])


def route(h, w, p, top):
    """[T, top] chosen experts (largest logits) and their weights (softmax over the chosen logits)."""
    z = lin(h, w[f"{p}.router"]) + d(w[f"{p}.router.b"])
    best, idx = torch.topk(z, top, dim=-1)
    return idx, torch.softmax(best, -1)


def experts_ff(h, w, p, f):
    idx, wt = route(h, w, p, int(f["router"]["top"]))
    out = torch.zeros_like(h)
    for e in range(int(f["router"]["experts"])):
        weight = (wt * (idx == e)).sum(-1, keepdim=True)
        out = out + weight * relu2_ff(h, w, f"{p}.e{e}")
    if f.get("shared"):
        out = out + torch.sigmoid(lin(h, w[f"{p}.shared.sg"])) * relu2_ff(h, w, f"{p}.shared")
    return out


# ------------------------------------------------------------------------------------------ the model
def hidden_states(cfg, w, tokens):
    """The residual stream after every layer, [layers, T, W]."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = layer_norm(d(w["embed"])[torch.as_tensor(tokens, dtype=torch.long)], w, "embed.norm", eps)
    out, kept = [], {}
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}", l["mixer"], l.get("mlp")
        h = layer_norm(x, w, f"{p}.norm1", eps)
        if l["type"] == "retention":
            y = retention(h, w, f"{p}.mix", m, eps)
        elif l["type"] == "wkv":
            y = wkv(h, w, f"{p}.mix", m, eps)
        elif l["type"] == "attention":
            if m.get("kv_from") is None:
                kept[i] = attention_kv(h, w, f"{p}.mix", m)
            y = diff_attention(h, w, f"{p}.mix", m, eps, kept[i if m.get("kv_from") is None else int(m["kv_from"])])
        else:
            raise ValueError(l["type"])
        x = x + mult * y
        if f is not None:
            h = layer_norm(x, w, f"{p}.norm2", eps)
            x = x + mult * (dense_ff(h, w, f"{p}.mlp") if f["kind"] == "dense" else experts_ff(h, w, f"{p}.mlp", f))
        out.append(x)
    return torch.stack(out)


def logits(cfg, w, tokens):
    """Logits at every position of one sequence, float64 [T, vocab]."""
    x = hidden_states(cfg, w, tokens)[-1]
    z = lin(layer_norm(x, w, "final.norm", float(cfg["norm"]["eps"])), w["head"])
    cap = cfg.get("logit_softcap")
    return z if not cap else float(cap) * torch.tanh(z / float(cap))


class PlainFedipel:
    """A model folder (config.json, model.safetensors) read without the engine's loader."""

    def __init__(self, model_dir):
        import json
        import struct
        from pathlib import Path

        import numpy as np
        model_dir = Path(model_dir)
        self.cfg = json.loads((model_dir / "config.json").read_text())
        raw = (model_dir / "model.safetensors").read_bytes()
        n = struct.unpack("<Q", raw[:8])[0]
        header = json.loads(raw[8:8 + n])
        self.w = {}
        for name, info in header.items():
            if name == "__metadata__":
                continue
            a, b = info["data_offsets"]
            data = raw[8 + n + a:8 + n + b]
            if info["dtype"] == "BF16":
                bits = np.frombuffer(data, dtype="<u2").astype(np.uint32) << 16
                t = torch.from_numpy(bits.view(np.float32).copy())
            elif info["dtype"] == "F32":
                t = torch.from_numpy(np.frombuffer(data, dtype="<f4").copy())
            else:
                raise ValueError(f"{name}: dtype {info['dtype']}")
            self.w[name] = t.reshape(info["shape"]).to(F64)

    def logits(self, tokens):
        return logits(self.cfg, self.w, tokens)

    def hidden_states(self, tokens):
        return hidden_states(self.cfg, self.w, tokens)

    def greedy(self, prompt, n):
        toks, out = list(prompt), []
        for _ in range(n):
            out.append(int(self.logits(toks)[-1].argmax()))
            toks.append(out[-1])
        return out
