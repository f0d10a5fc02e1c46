"""Gokosun as a plan: every layer has one layer norm (weight and bias) whose output the mixer and the feed-forward both read, and both are
added to the stream; mixers are a matrix memory with exponential gates (mLSTM), latent attention with a query latent and a learned sink per
head, or grouped attention with norms over the whole query and key projections and values mixed with those of the first layer that does so;
feed-forwards are gated with clamped halves, dense or as experts chosen by corrected sigmoid scores beside a shared expert.

Tensor names: `embed`, `l<i>.norm1` (with `.b`), `l<i>.mix.{q,k,v,g,o,norm,i,f}` (the gates i and f with `.b`), `l<i>.mix.{dq,dq.norm,uq,dkv,
dkv.norm,uk,uv,sink,o}` or `l<i>.mix.{q,k,v,q.norm,k.norm,vmix,o}`, `l<i>.mlp.{gate,up,down}` or `l<i>.mlp.{router, correction,
e<k>.{gate,up,down}, shared.{gate,up,down}}`, `final.norm`, `head`. They have no common root.
"""
from __future__ import annotations

from ..config.gokosun import GokosunConfig
from ..parts.plan import LayerPlan, ModelPlan, PartSpec, ScheduleEntry
from ..registry import register_architecture

MAX_POSITIONS = 1 << 20   # the rotations have no table: positions are bounded by the cache alone
GATE_SLOPE = 1.702        # slope of the sigmoid in the feed-forwards' gate


def gokosun_plan(c: GokosunConfig) -> ModelPlan:
    def norm(name):
        return PartSpec("layernorm", {"name": name, "size": c.width, "eps": c.norm_eps, "bias": "{}.b"})

    def rope(rot, pairing):
        return PartSpec("rope", {"rotary_dim": rot.dims, "theta": rot.base, "pairing": pairing, "yarn": rot.scaling}) if rot.dims else PartSpec("none")

    layers, ignored, first = [], [], c.first_mixed
    for i, l in enumerate(c.layers):
        m, p = l.mixer, f"l{i}"
        common = {"prefix": f"{p}.mix", "hidden": c.width, "heads": m.heads, "norm_eps": c.norm_eps}
        if l.type == "mlstm":
            mixer = PartSpec("mlstm", {**common, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap})
        elif l.type == "latent_attention":
            mixer = PartSpec("latent_attention", {**common, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "q_rank": m.q_rank, "scale": m.scale,
                                                  "position": rope(m.rot, "interleaved"), "sink": True})
        else:
            mix = None if not m.v_mix else ("first" if i == first else "mix")
            mixer = PartSpec("row_norm_attention", {**common, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "position": rope(m.rot, "half"),
                                                    "value_mix": mix})
            if mix != "mix":
                ignored.append(f"{p}.mix.vmix")
        f = l.mlp
        if f is None:
            ff = PartSpec("none")
        elif f.kind == "dense":
            ff = PartSpec("swiglu", {"prefix": f"{p}.mlp", "hidden": c.width, "intermediate": f.ff, "names": ("gate", "up", "down"), "clamp": (f.limit, GATE_SLOPE)})
        else:
            ff = PartSpec("routed_experts", {"prefix": f"{p}.mlp", "hidden": c.width, "expert_ff": f.ff, "experts": f.experts, "top": f.top, "route_scale": f.route_scale,
                                             "renorm": True, "shared_ff": f.shared_ff, "score": "sigmoid", "correction": "correction", "activation": "clamped_swiglu",
                                             "clamp": (f.limit, GATE_SLOPE), "shared_limit": f.shared_limit})
        layers.append(LayerPlan(prefix=p, block="parallel_sublayers", mixer=mixer, feed_forward=ff, mixer_norm=norm(f"{p}.norm1"), feed_forward_norm=PartSpec("none")))
    return ModelPlan(
        architecture="Gokosun", vocab_size=c.vocab, hidden_size=c.width, max_positions=MAX_POSITIONS,
        embedding=PartSpec("table", {"name": "embed", "vocab": c.vocab, "hidden": c.width}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))), final_norm=norm("final.norm"),
        head=PartSpec("linear", {"name": "head", "vocab": c.vocab, "hidden": c.width}),
        ignored_tensors=tuple(ignored), root="",
    )


register_architecture(["Gokosun", "gokosun"], GokosunConfig.from_dict, gokosun_plan,
                      traits={"attention": "mlstm+latent+row_norm", "qk_norm": True, "norm": "layernorm", "norm_unit_offset": False, "rope_style": "mixed",
                              "activation": "clamped_swiglu"})
