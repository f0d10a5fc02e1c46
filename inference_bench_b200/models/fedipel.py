"""Fedipel as a plan: pre-norm layers with layer norms (weight and bias) and a residual multiplier; mixers are retention (a linear
recurrence with a fixed decay per head and turned queries and keys), a recurrence with a decay per channel and token behind a token shift, or
differential attention over a window and the first tokens, which may read an earlier layer's keys and values; feed-forwards are dense SwiGLU
or experts with squared ReLUs, chosen by biased logits, beside a gated shared expert. The embedding is normed, the logits are capped.

Tensor names: `embed`, `embed.norm`, `l<i>.{norm1,norm2}` (norms with `.b`), `l<i>.mix.{q,k,v,g,o}`, `l<i>.mix.{mu.r,mu.k,mu.v,mu.g,mu.w,r,k,v,g,
w1,w2,w0,u,norm,o}` or `l<i>.mix.{q,k,v}` with `.b` biases and `l<i>.mix.{lq1,lk1,lq2,lk2,o}`, `l<i>.mlp.{gate,up,down}` or `l<i>.mlp.{router,
router.b, e<k>.{up,down}, shared.{up,down,sg}}`, `final.norm`, `head`. They have no common root.
"""
from __future__ import annotations

from ..config.fedipel import FedipelConfig
from ..parts.plan import LayerPlan, ModelPlan, PartSpec, ScheduleEntry
from ..registry import register_architecture

MAX_POSITIONS = 1 << 20   # the rotation has no table: positions are bounded by the cache alone


def fedipel_plan(c: FedipelConfig) -> ModelPlan:
    def norm(name):
        return PartSpec("layernorm", {"name": name, "size": c.width, "eps": c.norm_eps, "bias": "{}.b"})

    def rope(rot, pairing):
        return PartSpec("rope", {"rotary_dim": rot.dims, "theta": rot.base, "pairing": pairing}) if rot.dims else PartSpec("none")

    layers, schedule, ignored = [], [], []
    for i, l in enumerate(c.layers):
        m, p = l.mixer, f"l{i}"
        common = {"prefix": f"{p}.mix", "hidden": c.width, "heads": m.heads, "dim": m.dim, "norm_eps": c.norm_eps}
        kv_from = None
        if l.type == "retention":
            mixer = PartSpec("retention", {**common, "vdim": m.vdim, "decay": m.decay, "position": rope(m.rot, "half")})
        elif l.type == "wkv":
            mixer = PartSpec("wkv", common)
        else:
            kv_from = m.kv_from
            mixer = PartSpec("differential_attention", {**common, "kv_heads": m.kv_heads, "vdim": m.vdim, "scale": m.scale, "diff": m.diff,
                                                        "position": rope(m.rot, "interleaved"), "window": m.window, "keep_first": m.keep_first, "own_kv": kv_from is None})
            if kv_from is None:
                mixer.params["cache_window"], mixer.params["cache_keep"] = c.kept_keys(i)
        if l.mlp is None:
            ff, ff_norm = PartSpec("none"), PartSpec("none")
            ignored += [f"{p}.norm2", f"{p}.norm2.b"]
        else:
            f, ff_norm = l.mlp, norm(f"{p}.norm2")
            if f.kind == "dense":
                ff = PartSpec("swiglu", {"prefix": f"{p}.mlp", "hidden": c.width, "intermediate": f.ff, "names": ("gate", "up", "down")})
            else:
                ff = PartSpec("routed_experts", {"prefix": f"{p}.mlp", "hidden": c.width, "expert_ff": f.ff, "experts": f.experts, "top": f.top, "shared_ff": f.shared_ff,
                                                 "score": "chosen_softmax", "activation": "relu2", "router_bias": "router.b", "shared_gate": "sg"})
        layers.append(LayerPlan(prefix=p, block="prenorm", mixer=mixer, feed_forward=ff, mixer_norm=norm(f"{p}.norm1"), feed_forward_norm=ff_norm,
                                block_params=(("residual_mult", c.residual_mult),)))
        schedule.append(ScheduleEntry(i, cache_of=kv_from))   # one execution per layer, so a layer's number is its entry's
    return ModelPlan(
        architecture="Fedipel", vocab_size=c.vocab, hidden_size=c.width, max_positions=MAX_POSITIONS,
        embedding=PartSpec("table", {"name": "embed", "vocab": c.vocab, "hidden": c.width, "norm": norm("embed.norm")}),
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm("final.norm"),
        head=PartSpec("linear", {"name": "head", "vocab": c.vocab, "hidden": c.width, "softcap": c.logit_softcap}),
        ignored_tensors=tuple(ignored), root="",
    )


register_architecture(["Fedipel", "fedipel"], FedipelConfig.from_dict, fedipel_plan,
                      traits={"attention": "differential", "qk_norm": False, "norm": "layernorm", "norm_unit_offset": False, "rope_style": "interleaved", "activation": "relu2"})
