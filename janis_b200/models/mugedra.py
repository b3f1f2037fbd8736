"""Mugedra as an arrangement of parts.

A decoder whose layers are listed in the configuration: `PreNormBlock` with layer norms, a factor per feature on every
sublayer's result, and

* mixer: `ParallelMixers`, each branch's output normed and the two averaged (left to the kernel that adds them to the stream),
  over `left`, `TalkingHeadsAttention` without head mixing (normed and turned heads, frequencies along a ramp with their
  amplitude, capped scores, keys seen inside chunks, a gate per element), and `right`, `GatedDeltaRule`; both read one product
  of the input;
* feed-forward: `RoutedExperts` with sigmoid scores that are the weights themselves, on the experts' inputs; or none.

A run of layers may be passed several times: the schedule names it once a pass, each pass with cache lines of its own, and the
embedding's rows join the stream before every pass but the first.

Tensor names: `embed`, `l<i>.norm1|norm2|ls1|ls2`, `l<i>.mix.left.*`, `l<i>.mix.right.*`, `l<i>.mlp.*`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.mugedra import MugedraConfig
from ..engine.model import DecoderModel, LayerCall
from ..parts import registry as parts
from ..registry import register_architecture


def _attention(W, p, m, eps):
    position = parts.make("position", "rotary", head_dim=m.dim, base=m.rot_base, rotary_dims=m.rot_dims,
                          ramp_scaling=m.rot_scaling.to_dict() if m.rot_scaling is not None else None)
    names = {k: f"{p}.{k}" for k in ("q", "k", "v", "g", "o")}
    names.update(q_norm=f"{p}.q.norm", k_norm=f"{p}.k.norm")
    return parts.make("mixer", "talking_heads_attention", hidden=W, n_heads=m.heads, n_kv_heads=m.kv_heads, key_dim=m.dim,
                      value_dim=m.vdim, scale=m.scale, cap=m.softcap, block=m.chunk, head_norm_eps=eps, position=position, names=names)


def _delta_rule(W, p, m, eps):
    names = {k: f"{p}.{k}" for k in ("q", "k", "v", "g", "b", "a", "A_log", "dt_bias", "norm", "o")}
    names.update({f"{k}_conv": f"{p}.{k}.conv" for k in ("q", "k", "v")})
    return parts.make("mixer", "gated_delta_rule", hidden=W, n_heads=m.heads, n_key_heads=m.kv_heads, key_dim=m.dim, value_dim=m.vdim,
                      taps=m.conv, norm_eps=eps, names=names)


def build_mugedra(cfg: MugedraConfig) -> DecoderModel:
    W, eps = cfg.width, cfg.norm_eps

    def norm(name):
        return parts.make("norm", "layer_norm", width=W, eps=eps, weight_name=name)

    blocks = []
    unused = []                # what a folder may carry without its model using it
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}"
        m = layer.mixer
        mixer = parts.make("mixer", "parallel", hidden=W, eps=eps, deferred=True,
                           branches={"left": _attention(W, f"{p}.mix.left", m.left, eps),
                                     "right": _delta_rule(W, f"{p}.mix.right", m.right, eps)},
                           out_norm_names={k: f"{p}.mix.{k}.out" for k in ("left", "right")})
        ff = None
        if layer.mlp is not None:
            ff = parts.make("feed_forward", "routed_experts", hidden=W, n_experts=layer.mlp.experts, top=layer.mlp.top,
                            expert_ff=layer.mlp.expert_ff, limit=0.0, scale=1.0, act="silu", renormalize=False, weight_on="input",
                            names={"router": f"{p}.mlp.router", "expert": p + ".mlp.e{e}.{w}"})
        else:
            unused += [f"{p}.norm2", f"{p}.ls2"]
        blocks.append(parts.make("block", "pre_norm", mixer=mixer, feed_forward=ff, input_norm=norm(f"{p}.norm1"),
                                 pre_ff_norm=norm(f"{p}.norm2") if ff is not None else None, width=W, mixer_scale_name=f"{p}.ls1",
                                 ff_scale_name=f"{p}.ls2" if ff is not None else None))
    order = [(i, False) for i in range(len(blocks))]
    if cfg.loop is not None:
        lp = cfg.loop
        passes = [(i, turn > 0 and i == lp.start) for turn in range(lp.times) for i in range(lp.start, lp.stop)]
        order = order[:lp.start] + passes + order[lp.stop:]
    return DecoderModel(
        cfg,
        embedding=parts.make("embedding", "scaled_table", vocab=cfg.vocab, hidden=W, table_name="embed", scale=1.0,
                             init_std=1.0),
        blocks=blocks,
        final_norm=norm("final.norm"),
        head=parts.make("head", "capped_linear", vocab=cfg.vocab, hidden=W, table_name="head", softcap=0.0, init_std=W ** -0.5),
        schedule=[LayerCall(layer, line, add_embedding=again) for line, (layer, again) in enumerate(order)],
        ignorable_tensors=unused,
        max_context=1 << 20)


register_architecture("Mugedra", MugedraConfig, build_mugedra, model_types=("mugedra",), replace=True)
