"""Larulorn as an arrangement of parts.

A decoder whose layers are listed in the configuration, in the sandwich arrangement (`SandwichBlock`: a norm before and
after each sublayer) with plain RMS norms, each with one of two mixers and a dense feed-forward, a mixture of experts, or
none:

* "attention": `TalkingHeadsAttention` without head mixing, over all earlier keys: biases on the projections, rotary
  frequencies along a ramp with their amplitude, a learnt sink per head, and in layers that say so values mixed with those
  of the first such layer.
* "parallel": `ParallelMixers` that adds with constants, over `left`, `TalkingHeadsAttention` with plain rotary positions
  and a gate per element, and `right`, `GatedRecurrenceMixer`.
* feed-forward: `GatedMLP` with limits on gate and up, or `RoutedExperts` with softmax scores, groups scored by their best
  expert, plain squared-relu experts and a shared one without a gate.

Tensor names: `embed`, `l<i>.norm1|norm1b|norm2|norm2b`, `l<i>.mix.*` (a parallel layer's under `.left` and `.right`),
`l<i>.mlp.*`, `final.norm`, `head`.  The head is a table of its own whose logits are multiplied by `logit_scale`.
"""
from __future__ import annotations

from ..config.larulorn import LarulornConfig, PlainMoeSpec
from ..engine.model import DecoderModel, LayerCall
from ..parts import registry as parts
from ..registry import register_architecture


def _position(m):
    return parts.make("position", "rotary", head_dim=m.dim, base=m.rot_base, rotary_dims=m.rot_dims,
                      ramp_scaling=m.rot_scaling.to_dict() if m.rot_scaling is not None else None)


def _attention(W, p, m, value_mix):
    names = {k: f"{p}.{k}" for k in ("q", "k", "v", "o", "sink", "vmix")}
    names.update({f"{k}_bias": f"{p}.{k}.b" for k in ("q", "k", "v")})
    return parts.make("mixer", "talking_heads_attention", hidden=W, n_heads=m.heads, n_kv_heads=m.kv_heads, key_dim=m.dim,
                      value_dim=m.vdim, scale=m.scale, value_mix=value_mix, position=_position(m), names=names)


def _parallel(W, p, m):
    a, d = m.left, m.right
    left = parts.make("mixer", "talking_heads_attention", hidden=W, n_heads=a.heads, n_kv_heads=a.kv_heads, key_dim=a.dim,
                      value_dim=a.vdim, scale=a.scale, position=_position(a),
                      names={k: f"{p}.left.{k}" for k in ("q", "k", "v", "g", "o")})
    right = parts.make("mixer", "gated_recurrence", hidden=W, width=d.width, blocks=d.blocks, taps=d.conv,
                       names={**{k: f"{p}.right.{k}" for k in ("y", "x", "conv", "ra", "ri", "lam", "o")},
                              **{f"{k}_bias": f"{p}.right.{k}.b" for k in ("y", "x", "conv", "ra", "ri")}})
    return parts.make("mixer", "parallel", hidden=W, branches={"left": left, "right": right},
                      scales={"left": m.left_scale, "right": m.right_scale})


def _feed_forward(W, p, f):
    if isinstance(f, PlainMoeSpec):
        names = {"router": f"{p}.router", "expert": p + ".e{e}.{w}"}
        if f.shared_ff:
            names["shared"] = p + ".shared.{w}"
        return parts.make("feed_forward", "routed_experts", hidden=W, n_experts=f.experts, top=f.top, expert_ff=f.expert_ff,
                          limit=0.0, scale=1.0, group_count=f.group_count, group_keep=f.group_keep, group_score="best",
                          shared_ff=f.shared_ff, score="softmax", act="relu2", names=names)
    return parts.make("feed_forward", "gated_mlp", hidden=W, intermediate=f.ff, act="clamped_swish", limit=f.limit,
                      names={k: f"{p}.{k}" for k in ("gate", "up", "down")})


def build_larulorn(cfg: LarulornConfig) -> DecoderModel:
    W = cfg.width

    def norm(name):
        return parts.make("norm", "rms_norm", width=W, eps=cfg.norm_eps, weight_name=name, init_mean=1.0)

    blocks = []
    unused = []                # what a folder may carry without its model using it
    first_mixed = next((i for i, l in enumerate(cfg.layers) if l.type == "attention" and l.mixer.v_mix), None)
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}"
        if layer.type == "attention":
            mix = None if not layer.mixer.v_mix else ("first" if i == first_mixed else "mix")
            if mix != "mix":
                unused.append(f"{p}.mix.vmix")
            mixer = _attention(W, f"{p}.mix", layer.mixer, mix)
        else:
            mixer = _parallel(W, f"{p}.mix", layer.mixer)
        ff = _feed_forward(W, f"{p}.mlp", layer.mlp) if layer.mlp is not None else None
        if ff is None:
            unused += [f"{p}.norm2", f"{p}.norm2b"]
        blocks.append(parts.make("block", "sandwich", mixer=mixer, feed_forward=ff, input_norm=norm(f"{p}.norm1"),
                                 post_mixer_norm=norm(f"{p}.norm1b"), pre_ff_norm=norm(f"{p}.norm2") if ff is not None else None,
                                 post_ff_norm=norm(f"{p}.norm2b") if ff is not None else None))
    return DecoderModel(
        cfg,
        embedding=parts.make("embedding", "scaled_table", vocab=cfg.vocab, hidden=W, table_name="embed", scale=1.0,
                             init_std=1.0),
        blocks=blocks,
        final_norm=norm("final.norm"),
        head=parts.make("head", "capped_linear", vocab=cfg.vocab, hidden=W, table_name="head", softcap=0.0,
                        scale=cfg.logit_scale, init_std=W ** -0.5),
        schedule=[LayerCall(i, i) for i in range(len(blocks))],
        ignorable_tensors=unused,
        max_context=1 << 20)


register_architecture("Larulorn", LarulornConfig, build_larulorn, model_types=("larulorn",), replace=True)
