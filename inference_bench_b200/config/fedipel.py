"""Typed configuration of the Fedipel decoder, read from its own config.json keys.

A Fedipel model is a list of layers, each with a mixer (retention, a recurrence with a data-dependent decay, or differential attention over a
window and the first tokens) and a feed-forward that is dense, a mixture of experts, or absent. config.json gives every size and constant but
the inner size of the recurrence's decay, which is its tensors' own; nothing here fixes one.

    architecture    "Fedipel"
    vocab, width    vocabulary size and width of the residual stream
    norm.eps        epsilon of every norm
    residual_mult   factor on every sublayer's output before it is added to the stream
    logit_softcap   c of logits <- c tanh(logits / c); null: logits as they are
    layers[i]       type "retention": mixer {heads, dim, vdim, decay [heads], rot {base, dims}}
                    type "wkv":       mixer {heads, dim}
                    type "attention": mixer {heads, kv_heads, dim, vdim, scale, diff, mask {size, keep_first} | null, rot {base, dims}, kv_from?}
                    mlp null | {kind "dense", ff} | {kind "moe", expert {ff}, router {experts, top}, shared {ff}?}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional

from . import ConfigError

MIXER_TYPES = ("retention", "wkv", "attention")
MLP_KINDS = ("dense", "moe")


def _need(d: Mapping[str, Any], key: str, where: str):
    if not isinstance(d, Mapping) or d.get(key) is None:
        raise ConfigError(f"config.json has no {where}.{key}")
    return d[key]


def _sizes(c, names, where: str) -> None:
    for name in names:
        if getattr(c, name) <= 0:
            raise ConfigError(f"{where}.{name} must be positive, got {getattr(c, name)}")


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int       # how many of a head's (or map's) first entries are turned

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], dim: int, where: str) -> "Rotation":
        r = m.get("rot")
        c = cls(1.0, 0) if r is None else cls(float(_need(r, "base", where + ".rot")), int(_need(r, "dims", where + ".rot")))
        if c.dims < 0 or c.dims % 2 or c.dims > dim or not c.base > 0:
            raise ConfigError(f"{where}.rot: dims {c.dims} must be even and at most dim {dim}, base {c.base} positive")
        return c

    def to_dict(self) -> dict[str, Any]:
        return {"base": self.base, "dims": self.dims}


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: tuple        # one a head
    rot: Rotation

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "RetentionConfig":
        heads, dim, vdim = (int(_need(m, k, where)) for k in ("heads", "dim", "vdim"))
        decay = _need(m, "decay", where)
        decay = tuple(float(d) for d in (decay if isinstance(decay, (list, tuple)) else [decay] * heads))
        c = cls(heads, dim, vdim, decay, Rotation.from_dict(m, dim, where))
        _sizes(c, ("heads", "dim", "vdim"), where)
        if c.dim > 512:
            raise ConfigError(f"{where}.dim {c.dim} is above 512")
        if len(c.decay) != c.heads or any(not 0.0 <= d <= 1.0 for d in c.decay):
            raise ConfigError(f"{where}.decay must give {c.heads} numbers in [0, 1], got {list(c.decay)}")
        return c

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay), "rot": self.rot.to_dict()}


@dataclass(frozen=True)
class WkvConfig:
    heads: int
    dim: int

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "WkvConfig":
        c = cls(int(_need(m, "heads", where)), int(_need(m, "dim", where)))
        _sizes(c, ("heads", "dim"), where)
        if c.dim > 512:
            raise ConfigError(f"{where}.dim {c.dim} is above 512")
        return c

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim}


@dataclass(frozen=True)
class DiffAttentionConfig:
    heads: int
    kv_heads: int
    dim: int                        # size of one map of a query or key head
    vdim: int
    scale: float
    diff: float
    window: Optional[int]           # a position sees itself and the window - 1 before it; None: every earlier position
    keep_first: int                 # with a window: the positions 0 .. keep_first - 1 are seen as well
    rot: Rotation
    kv_from: Optional[int] = None   # the layer whose cached keys and values this layer reads instead of making its own

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "DiffAttentionConfig":
        mask = m.get("mask")
        dim = int(_need(m, "dim", where))
        c = cls(heads=int(_need(m, "heads", where)), kv_heads=int(m.get("kv_heads") or m["heads"]), dim=dim, vdim=int(_need(m, "vdim", where)),
                scale=float(_need(m, "scale", where)), diff=float(_need(m, "diff", where)),
                window=None if mask is None else int(_need(mask, "size", where + ".mask")), keep_first=0 if mask is None else int(mask.get("keep_first") or 0),
                rot=Rotation.from_dict(m, dim, where), kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
        _sizes(c, ("heads", "kv_heads", "dim", "vdim"), where)
        if c.heads % c.kv_heads:
            raise ConfigError(f"{where}: {c.heads} heads are not a multiple of {c.kv_heads} kv_heads")
        if max(2 * c.dim, c.vdim) > 256:
            raise ConfigError(f"{where}: two maps of {c.dim} and values of {c.vdim}: at most 256 are built")
        if (c.window is not None and c.window <= 0) or c.keep_first < 0:
            raise ConfigError(f"{where}.mask: size {c.window} must be positive, keep_first {c.keep_first} not negative")
        return c

    def to_dict(self) -> dict[str, Any]:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale, "diff": self.diff,
             "mask": None if self.window is None else {"size": self.window, "keep_first": self.keep_first}, "rot": self.rot.to_dict()}
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        return d


MIXERS = {"retention": RetentionConfig, "wkv": WkvConfig, "attention": DiffAttentionConfig}


@dataclass(frozen=True)
class FedipelMlp:
    kind: str               # "dense" | "moe"
    ff: int                 # dense: the inner size; moe: one expert's
    experts: int = 0
    top: int = 0
    shared_ff: int = 0      # 0: no shared expert

    @classmethod
    def from_dict(cls, f: Mapping[str, Any], where: str) -> "FedipelMlp":
        kind = _need(f, "kind", where)
        if kind == "dense":
            c = cls("dense", int(_need(f, "ff", where)))
        elif kind == "moe":
            r = _need(f, "router", where)
            shared = f.get("shared")
            c = cls("moe", int(_need(_need(f, "expert", where), "ff", where + ".expert")), int(_need(r, "experts", where + ".router")), int(_need(r, "top", where + ".router")),
                    0 if not shared else int(_need(shared, "ff", where + ".shared")))
            if c.experts <= 0 or not 0 < c.top <= c.experts:
                raise ConfigError(f"{where}.router: top {c.top} of {c.experts} experts")
        else:
            raise ConfigError(f"{where}.kind {kind!r} is not supported (known: {', '.join(MLP_KINDS)})")
        if c.ff <= 0 or c.shared_ff < 0:
            raise ConfigError(f"{where}: inner sizes must be positive")
        return c

    def to_dict(self) -> dict[str, Any]:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        d: dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


@dataclass(frozen=True)
class FedipelLayer:
    type: str
    mixer: Any              # RetentionConfig | WkvConfig | DiffAttentionConfig
    mlp: Optional[FedipelMlp]


@dataclass(frozen=True)
class FedipelConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    logit_softcap: Optional[float]
    layers: tuple
    architecture: str = "Fedipel"

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def kept_keys(self, i: int) -> tuple:
        """(window or None, first positions) that the cache of attention layer i has to hold: what the layer itself and every layer that reads its
        cache see."""
        masks = [l.mixer for j, l in enumerate(self.layers) if l.type == "attention" and (j == i or l.mixer.kv_from == i)]
        window = None if any(m.window is None for m in masks) else max(m.window for m in masks)
        return window, (max(m.keep_first for m in masks) if window else 0)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "FedipelConfig":
        layers_raw = _need(raw, "layers", "config")
        if not isinstance(layers_raw, (list, tuple)) or not layers_raw:
            raise ConfigError("config.json: layers must be a non-empty list")
        layers = []
        for i, l in enumerate(layers_raw):
            t = _need(l, "type", f"layers[{i}]")
            if t not in MIXERS:
                raise ConfigError(f"layers[{i}].type {t!r} is not supported (known: {', '.join(MIXER_TYPES)})")
            mixer = MIXERS[t].from_dict(_need(l, "mixer", f"layers[{i}]"), f"layers[{i}].mixer")
            layers.append(FedipelLayer(t, mixer, None if l.get("mlp") is None else FedipelMlp.from_dict(l["mlp"], f"layers[{i}].mlp")))
        for i, l in enumerate(layers):
            j = l.mixer.kv_from if l.type == "attention" else None
            if j is None:
                continue
            if not 0 <= j < i or layers[j].type != "attention":
                raise ConfigError(f"layers[{i}].mixer.kv_from = {j} does not name an earlier attention layer")
            o, m = layers[j].mixer, l.mixer
            if o.kv_from is not None:
                raise ConfigError(f"layers[{i}].mixer.kv_from = {j}, but layer {j} has no keys and values of its own")
            if (o.kv_heads, o.dim, o.vdim, o.rot) != (m.kv_heads, m.dim, m.vdim, m.rot):
                raise ConfigError(f"layers[{i}].mixer reads layer {j}'s keys and values, but their kv_heads, dim, vdim or rotation differ")
        cfg = cls(vocab=int(_need(raw, "vocab", "config")), width=int(_need(raw, "width", "config")),
                  norm_eps=float(_need(_need(raw, "norm", "config"), "eps", "norm")), residual_mult=float(raw.get("residual_mult", 1.0)),
                  logit_softcap=None if raw.get("logit_softcap") is None else float(raw["logit_softcap"]), layers=tuple(layers),
                  architecture=str(raw.get("architecture", "Fedipel")))
        if cfg.vocab <= 0 or cfg.width <= 0 or not cfg.norm_eps > 0:
            raise ConfigError(f"vocab {cfg.vocab}, width {cfg.width} and norm.eps {cfg.norm_eps} must be positive")
        if cfg.logit_softcap is not None and not cfg.logit_softcap > 0:
            raise ConfigError(f"logit_softcap must be positive, got {cfg.logit_softcap}")
        return cfg

    def to_dict(self) -> dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
                "logit_softcap": self.logit_softcap,
                "layers": [{"type": l.type, "mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict()} for l in self.layers]}
