"""A plain, slow Gokosun: one function per mechanism, written from the architecture's equations in double precision with torch on the
CPU. It shares no code with the engine and is what the engine's kernels are compared with.

Notation: x [T, W] is one sequence's residual stream (rows are positions 0..T-1), `cfg` the dictionary of config.json, `w` a dictionary
name -> tensor (any floating dtype; everything is widened to float64).

    x = embed[tokens];   per layer  h = LN(x),  x = x + mixer(h) + ff(h)   (a layer may have no feed-forward);   logits = head LN(x)
LN is a layer norm with a weight and a bias; mixers are a matrix memory with exponential gates, latent attention with a sink, or grouped
attention with whole-projection norms and mixed values; feed-forwards are gated with clamped halves, dense or as routed experts.
"""
from __future__ import annotations

import contextlib
import math

import torch

F64 = torch.float64

ROUND = False     # True (`rounded`): what a bfloat16 engine stores in 16 bits is rounded: the inputs of every matrix product, turned queries and keys,
                  # values, cached latents, attention outputs. How far that moves a row says how far an engine's own rounding may.


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


def yarn_frequencies(dims, base, scaling):
    """The dims/2 rotation frequencies and the factor on cosines and sines. Without `scaling`: base^(-2i/dims) and 1. With it (factor, original,
    fast, slow) pair i keeps its frequency below a ramp of pairs, has it divided by `factor` above, and a blend of both on the ramp, whose ends
    are the pairs that turn `fast` and `slow` times over `original` positions."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=F64), 1.0
    factor = float(scaling["factor"])

    def pair_of(turns):
        return dims * math.log(float(scaling["original"]) / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(pair_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(pair_of(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(factor) + 1.0


def rotate(x, positions, rot, interleaved):
    """x [T, heads, n]: the first rot["dims"] entries are turned in pairs; pair i is (i, i + dims/2), or (2i, 2i + 1) when interleaved."""
    dims = int(rot["dims"]) if rot else 0
    n = dims // 2
    if n == 0:
        return x
    f, amp = yarn_frequencies(dims, float(rot["base"]), rot.get("scaling"))
    a = d(positions)[:, None, None] * f
    cos, sin = torch.cos(a) * amp, torch.sin(a) * amp
    if interleaved:
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        turned = torch.stack([u * cos - v * sin, v * cos + u * sin], -1).flatten(-2)
    else:
        u, v = x[..., :n], x[..., n:dims]
        turned = torch.cat([u * cos - v * sin, v * cos + u * sin], -1)
    return torch.cat([turned, x[..., dims:]], -1)


def causal_softmax(s, sink=None):
    """s [T, T] scores; row i sees j <= i. sink: a score without key or value that only the denominator holds."""
    T = s.shape[0]
    s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], -math.inf)
    if sink is None:
        return torch.softmax(s, -1)
    return torch.softmax(torch.cat([s, torch.full((T, 1), float(sink), dtype=F64)], -1), -1)[:, :T]


# ------------------------------------------------------------------------------------------ the matrix memory
def memory_scan(q, k, v, i, f):
    """q, k [T, H, D], v [T, H, V], log input gates i and log forget gates f [T, H]:
    m_t = max(f + m, i) from m = 0;  S_t = e^(f + m_(t-1) - m_t) S + e^(i - m_t) k v^T, n_t likewise with k;
    o_t = S_t^T q / (max(|n_t . q|, e^(-m_t)) + 1e-6)."""
    T, H, D = q.shape
    S, n, m = torch.zeros((H, D, v.shape[2]), dtype=F64), torch.zeros((H, D), dtype=F64), torch.zeros(H, dtype=F64)
    o = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + take[:, None, None] * (k[t][:, :, None] * v[t][:, None, :])
        n = keep[:, None] * n + take[:, None] * k[t]
        m = new
        norm = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        o[t] = (S * q[t][:, :, None]).sum(1) / norm[:, None]
    return o


def memory_gates(h, w, p, cap):
    """(log input gates, log forget gates), both [T, heads]."""
    def capped(s):
        return cap * torch.tanh((lin(h, w[f"{p}.{s}"]) + d(w[f"{p}.{s}.b"])) / cap)
    return capped("i"), torch.nn.functional.logsigmoid(capped("f"))


def memory(h, w, p, m, eps):
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = lin(h, w[f"{p}.q"]).view(T, H, D) / math.sqrt(D)
    k, v = lin(h, w[f"{p}.k"]).view(T, H, D), lin(h, w[f"{p}.v"]).view(T, H, V)
    i, f = memory_gates(h, w, p, float(m["gate_cap"]))
    o = rms_unit(memory_scan(q, k, v, i, f), eps).reshape(T, H * V)
    return lin(o * d(w[f"{p}.norm"]) * torch.sigmoid(lin(h, w[f"{p}.g"])), w[f"{p}.o"])


# ------------------------------------------------------------------------------------------ latent attention
def latent_attention(h, w, p, m, eps):
    T = h.shape[0]
    H, D, R, V, K = (int(m[s]) for s in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    pos = torch.arange(T)
    cq = rms_unit(lin(h, w[f"{p}.dq"]), eps) * d(w[f"{p}.dq.norm"])
    q = lin(cq, w[f"{p}.uq"]).view(T, H, D + R)
    down = lin(h, w[f"{p}.dkv"])
    c = rnd(rms_unit(down[:, :K], eps) * d(w[f"{p}.dkv.norm"]))
    kr = rnd(rotate(down[:, None, K:], pos, m["rot"], True)[:, 0])
    qr = rnd(rotate(q[:, :, D:], pos, m["rot"], True))
    k, v = lin(c, w[f"{p}.uk"]).view(T, H, D), lin(c, w[f"{p}.uv"]).view(T, H, V)
    out = torch.zeros((T, H, V), dtype=F64)
    for a in range(H):
        s = (rnd(q[:, a, :D]) @ k[:, a].T + qr[:, a] @ kr.T) * float(m["scale"])
        out[:, a] = causal_softmax(s, d(w[f"{p}.sink"])[a]) @ v[:, a]
    return lin(out.reshape(T, H * V), w[f"{p}.o"])


# ------------------------------------------------------------------------------------------ grouped attention
def mixed_values(v, first, w, p):
    """The values of a layer that mixes them: its own where it is the first such layer (`first` None), else a blend with the first one's."""
    if first is None:
        return v
    lam = d(w[f"{p}.vmix"]).reshape(())
    return (1.0 - lam) * v + lam * first


def attention(h, w, p, m, eps, first):
    """Returns (output, the layer's own values as projected)."""
    T = h.shape[0]
    H, G, D, V = (int(m[s]) for s in ("heads", "kv_heads", "dim", "vdim"))
    pos = torch.arange(T)
    q = rms_unit(lin(h, w[f"{p}.q"]), eps) * d(w[f"{p}.q.norm"])
    k = rms_unit(lin(h, w[f"{p}.k"]), eps) * d(w[f"{p}.k.norm"])
    q, k = rnd(rotate(q.view(T, H, D), pos, m["rot"], False)), rnd(rotate(k.view(T, G, D), pos, m["rot"], False))
    own = lin(h, w[f"{p}.v"])
    v = rnd(mixed_values(own, first, w, p) if m.get("v_mix") else own).view(T, G, V)
    out = torch.zeros((T, H, V), dtype=F64)
    for a in range(H):
        b = a // (H // G)
        out[:, a] = causal_softmax((q[:, a] @ k[:, b].T) * float(m["scale"])) @ v[:, b]
    return lin(out.reshape(T, H * V), w[f"{p}.o"]), own


# ------------------------------------------------------------------------------------------ feed-forwards
def clamped_glu(g, u, limit):
    """g' sigmoid(1.702 g') (u' + 1) with g' = min(g, limit), u' = u cut to [-limit, limit]."""
    g, u = torch.clamp(g, max=limit), torch.clamp(u, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def gated_ff(h, w, p, limit):
    return lin(clamped_glu(lin(h, w[f"{p}.gate"]), lin(h, w[f"{p}.up"]), limit), w[f"{p}.down"])


def route(h, w, p, top, scale):
    """[T, top] chosen experts (largest sigmoid score plus correction) and their weights (scores alone, divided by their sum, times scale)."""
    s = torch.sigmoid(lin(h, w[f"{p}.router"]))
    idx = torch.topk(s + d(w[f"{p}.correction"]), top, dim=-1).indices
    wt = torch.gather(s, 1, idx)
    return idx, wt / (wt.sum(-1, keepdim=True) + 1e-20) * scale


def experts_ff(h, w, p, f):
    r = f["router"]
    idx, wt = route(h, w, p, int(r["top"]), float(r["scale"]))
    out = torch.zeros_like(h)
    for e in range(int(r["experts"])):
        out = out + (wt * (idx == e)).sum(-1, keepdim=True) * gated_ff(h, w, f"{p}.e{e}", float(f["expert"]["limit"]))
    if f.get("shared"):
        out = out + gated_ff(h, w, f"{p}.shared", float(f["shared"]["limit"]))
    return out


# ------------------------------------------------------------------------------------------ the model
def hidden_states(cfg, w, tokens):
    """The residual stream after every layer, [layers, T, W]."""
    return hidden_from(cfg, w, d(w["embed"])[torch.as_tensor(tokens, dtype=torch.long)])


def hidden_from(cfg, w, x):
    """The same from the stream in front of the first layer."""
    eps = float(cfg["norm"]["eps"])
    out, first = [], None
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.mix", l["mixer"], l.get("mlp")
        h = layer_norm(x, w, f"l{i}.norm1", eps)
        if l["type"] == "mlstm":
            y = memory(h, w, p, m, eps)
        elif l["type"] == "latent_attention":
            y = latent_attention(h, w, p, m, eps)
        elif l["type"] == "attention":
            y, own = attention(h, w, p, m, eps, first)
            if m.get("v_mix") and first is None:
                first = own
        else:
            raise ValueError(l["type"])
        if f is not None:
            y = y + (gated_ff(h, w, f"l{i}.mlp", float(f["limit"])) if f["kind"] == "dense" else experts_ff(h, w, f"l{i}.mlp", f))
        x = x + y
        out.append(x)
    return torch.stack(out)


def logits(cfg, w, tokens):
    """Logits at every position of one sequence, float64 [T, vocab]."""
    return lin(layer_norm(hidden_states(cfg, w, tokens)[-1], w, "final.norm", float(cfg["norm"]["eps"])), w["head"])


class PlainGokosun:
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
        self.w = {}
        for name, info in json.loads(raw[8:8 + n]).items():
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
