"""Typed configuration of the Gokosun decoder, read from its own config.json keys.

A Gokosun model is a list of layers, each with a mixer (a matrix memory with exponential gates, latent attention with a sink, or grouped
attention whose values may be mixed with an earlier layer's) and beside it, on the same normed input, a feed-forward that is dense, a mixture
of experts, or absent. config.json gives every size and every constant that differs between models.

    architecture    "Gokosun"
    vocab, width    vocabulary size and width of the residual stream
    norm.eps        epsilon of every norm
    layers[i]       type "mlstm":            mixer {heads, dim, vdim, gate_cap}
                    type "latent_attention": mixer {heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot {base, dims, scaling?}}
                    type "attention":        mixer {heads, kv_heads, dim, vdim, scale, v_mix, rot {base, dims, scaling?}}
                    mlp null | {kind "dense", ff, limit} | {kind "moe", expert {ff, limit}, router {experts, top, scale}, shared {ff, limit}?}
    rot.scaling     {factor, original, fast, slow}: the rotation's frequencies are rescaled (parts/standard.py)
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional

from . import ConfigError

MIXER_TYPES = ("mlstm", "latent_attention", "attention")
MLP_KINDS = ("dense", "moe")
MAX_KEY_DIM = 512    # a memory head's key size the recurrence kernel holds
MAX_HEAD_DIM = 256   # a grouped attention head's size


def _need(d: Mapping[str, Any], key: str, where: str):
    if not isinstance(d, Mapping) or d.get(key) is None:
        raise ConfigError(f"config.json has no {where}.{key}")
    return d[key]


def _sizes(c, names, where: str) -> None:
    for name in names:
        if not getattr(c, name) > 0:
            raise ConfigError(f"{where}.{name} must be positive, got {getattr(c, name)}")


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int                          # how many of the rotated part's first entries are turned
    scaling: Optional[tuple] = None    # (factor, original, fast, slow)

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], dim: int, where: str) -> "Rotation":
        r = m.get("rot")
        if r is None:
            return cls(1.0, 0)
        s = r.get("scaling")
        scaling = None if not s else tuple(float(_need(s, k, where + ".rot.scaling")) for k in ("factor", "original", "fast", "slow"))
        c = cls(float(_need(r, "base", where + ".rot")), int(_need(r, "dims", where + ".rot")), scaling)
        if c.dims < 0 or c.dims % 2 or c.dims > dim or not c.base > 0:
            raise ConfigError(f"{where}.rot: dims {c.dims} must be even and at most {dim}, base {c.base} positive")
        if scaling is not None and (min(scaling) <= 0 or c.base == 1.0):
            raise ConfigError(f"{where}.rot.scaling {list(scaling)} must be positive numbers (and base not 1)")
        return c

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = dict(zip(("factor", "original", "fast", "slow"), self.scaling))
        return d


@dataclass(frozen=True)
class MemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "MemoryConfig":
        c = cls(*(int(_need(m, k, where)) for k in ("heads", "dim", "vdim")), float(_need(m, "gate_cap", where)))
        _sizes(c, ("heads", "dim", "vdim", "gate_cap"), where)
        if c.dim > MAX_KEY_DIM:
            raise ConfigError(f"{where}.dim {c.dim} is above {MAX_KEY_DIM}")
        return c

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "gate_cap": self.gate_cap}


@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int          # unrotated part of a query or key head
    rot_dim: int      # rotated part
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot: Rotation

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "LatentConfig":
        heads, dim, rot_dim, vdim, kv_rank, q_rank = (int(_need(m, k, where)) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
        c = cls(heads, dim, rot_dim, vdim, kv_rank, q_rank, float(_need(m, "scale", where)), Rotation.from_dict(m, rot_dim, where))
        _sizes(c, ("heads", "dim", "vdim", "kv_rank", "q_rank"), where)
        if c.rot_dim < 0:
            raise ConfigError(f"{where}.rot_dim {c.rot_dim} must not be negative")
        return c

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank, "q_rank": self.q_rank, "scale": self.scale,
                "rot": self.rot.to_dict()}


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    v_mix: bool       # values are mixed with those of the first layer that has this set
    rot: Rotation

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "AttentionConfig":
        heads, dim, vdim = (int(_need(m, k, where)) for k in ("heads", "dim", "vdim"))
        c = cls(heads, int(m.get("kv_heads") or heads), dim, vdim, float(_need(m, "scale", where)), bool(m.get("v_mix", False)), Rotation.from_dict(m, dim, where))
        _sizes(c, ("heads", "kv_heads", "dim", "vdim"), where)
        if c.heads % c.kv_heads:
            raise ConfigError(f"{where}: {c.heads} heads are not a multiple of {c.kv_heads} kv_heads")
        if max(c.dim, c.vdim) > MAX_HEAD_DIM:
            raise ConfigError(f"{where}: heads of {c.dim} and {c.vdim}: at most {MAX_HEAD_DIM} are built")
        return c

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale, "v_mix": self.v_mix, "rot": self.rot.to_dict()}


MIXERS = {"mlstm": MemoryConfig, "latent_attention": LatentConfig, "attention": AttentionConfig}


@dataclass(frozen=True)
class GokosunMlp:
    kind: str                   # "dense" | "moe"
    ff: int                     # dense: the inner size; moe: one expert's
    limit: float
    experts: int = 0
    top: int = 0
    route_scale: float = 1.0
    shared_ff: int = 0          # 0: no shared expert
    shared_limit: float = 0.0

    @classmethod
    def from_dict(cls, f: Mapping[str, Any], where: str) -> "GokosunMlp":
        kind = _need(f, "kind", where)
        if kind == "dense":
            c = cls("dense", int(_need(f, "ff", where)), float(_need(f, "limit", where)))
        elif kind == "moe":
            r, e, s = _need(f, "router", where), _need(f, "expert", where), f.get("shared")
            c = cls("moe", int(_need(e, "ff", where + ".expert")), float(_need(e, "limit", where + ".expert")), int(_need(r, "experts", where + ".router")),
                    int(_need(r, "top", where + ".router")), float(r.get("scale", 1.0)), 0 if not s else int(_need(s, "ff", where + ".shared")),
                    0.0 if not s else float(_need(s, "limit", where + ".shared")))
            if c.experts <= 0 or not 0 < c.top <= c.experts:
                raise ConfigError(f"{where}.router: top {c.top} of {c.experts} experts")
        else:
            raise ConfigError(f"{where}.kind {kind!r} is not supported (known: {', '.join(MLP_KINDS)})")
        if c.ff <= 0 or c.shared_ff < 0:
            raise ConfigError(f"{where}: inner sizes must be positive")
        if not c.limit > 0 or (c.shared_ff and not c.shared_limit > 0):
            raise ConfigError(f"{where}: limits must be positive, got {c.limit} and {c.shared_limit}")
        return c

    def to_dict(self) -> dict[str, Any]:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff, "limit": self.limit}
        d: dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit}, "router": {"experts": self.experts, "top": self.top, "scale": self.route_scale}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff, "limit": self.shared_limit}
        return d


@dataclass(frozen=True)
class GokosunLayer:
    type: str
    mixer: Any              # MemoryConfig | LatentConfig | AttentionConfig
    mlp: Optional[GokosunMlp]


@dataclass(frozen=True)
class GokosunConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple
    architecture: str = "Gokosun"

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def first_mixed(self) -> Optional[int]:
        """The layer whose values the other layers with v_mix mix theirs with."""
        return next((i for i, l in enumerate(self.layers) if l.type == "attention" and l.mixer.v_mix), None)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "GokosunConfig":
        layers_raw = _need(raw, "layers", "config")
        if not isinstance(layers_raw, (list, tuple)) or not layers_raw:
            raise ConfigError("config.json: layers must be a non-empty list")
        layers = []
        for i, l in enumerate(layers_raw):
            t = _need(l, "type", f"layers[{i}]")
            if t not in MIXERS:
                raise ConfigError(f"layers[{i}].type {t!r} is not supported (known: {', '.join(MIXER_TYPES)})")
            mixer = MIXERS[t].from_dict(_need(l, "mixer", f"layers[{i}]"), f"layers[{i}].mixer")
            layers.append(GokosunLayer(t, mixer, None if l.get("mlp") is None else GokosunMlp.from_dict(l["mlp"], f"layers[{i}].mlp")))
        cfg = cls(vocab=int(_need(raw, "vocab", "config")), width=int(_need(raw, "width", "config")), norm_eps=float(_need(_need(raw, "norm", "config"), "eps", "norm")),
                  layers=tuple(layers), architecture=str(raw.get("architecture", "Gokosun")))
        if cfg.vocab <= 0 or cfg.width <= 0 or not cfg.norm_eps > 0:
            raise ConfigError(f"vocab {cfg.vocab}, width {cfg.width} and norm.eps {cfg.norm_eps} must be positive")
        first = cfg.first_mixed
        for i, l in enumerate(layers):
            if l.type == "attention" and l.mixer.v_mix and l.mixer.kv_heads * l.mixer.vdim != layers[first].mixer.kv_heads * layers[first].mixer.vdim:
                raise ConfigError(f"layers[{i}].mixer mixes its values with layer {first}'s, but has {l.mixer.kv_heads * l.mixer.vdim} instead of "
                                  f"{layers[first].mixer.kv_heads * layers[first].mixer.vdim} a token")
        return cfg

    def to_dict(self) -> dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "layers": [{"type": l.type, "mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict()} for l in self.layers]}
