"""Softmax attention whose heads are mixed before the softmax, with values of a size of their own.

With H query heads over G key/value heads (query head h uses key/value head h // (H/G)), keys of d features
and values of dv:

    raw_g[i, j] = (q_g[i] . k[j]) * scale                     positions encoded on q and k by `position`
    s_h[i, j]   = sum_g M[h, g] raw_g[i, j]                   M: a stored H x H matrix (names["talk"]; absent: none)
    p_h[i, j]   = exp(s_h[i, j]) / (sink + sum_j' exp(s_h[i, j']))
    o_h[i]      = sum_j p_h[i, j] v[j]

over the keys j <= i that lie in the query's block of `block` positions (block 0: all of them; blocks are counted
from the sequence's first position) and, with a `window`, among the query's last `window` positions (i - j < window:
the query's own and the window - 1 before it).  `sink` adds 1 to the denominator: a key of score 0 that has no value.  With a
`value_position` the values are rotated by their own position before they are cached (over all dv features) and
each head's output is turned back by the query's position, so that o depends on relative positions only.

With a gate (names["g"]) the heads side by side are multiplied, element by element, by sigmoid(Wg y) before the
output projection; Wg's rows stand behind the other projections' in the one product.

Further options.  `values_from_keys`: there is no value projection; a key/value head's values are its keys as
projected, before any turn or norm (so the value size is the key size), cached beside the keys.  `unit_norm_eps`:
after the turn every head of q and k is divided by its own root mean square, sqrt(mean(head^2) + eps), without a
weight.  A position encoding of pairs="neighbours" turns (2i, 2i + 1) instead of (i, i + rot/2).  `keep_first` (with
a window): the sequence's first `keep_first` positions stay seen behind the window, at their true positions.
`gate="head"`: Wg has one row per head and the gate is one number per head.  Biases on the projections (names
["q_bias"], ["k_bias"], ["v_bias"], all three or none) are added before the turn.  A learnt sink (names["sink"], a number
per head): exp(sink_h) joins the denominator instead of 1.  The position encoding's amplitude multiplies sine and cosine.
`value_mix`: "first" leaves the layer's values where later layers of the step find them, "mix" makes the values
(1 - m) v + m v_first with the stored number m (names["vmix"]) before they are cached, v_first being the values of the
same token in the layer that left them.

`head_norm_eps` with names["q_norm"] and names["k_norm"]: every head of q and k is divided by sqrt(mean(head^2) + eps) and
multiplied by a stored weight of d features (one for all heads of q, one for those of k) before it turns.  `cap`: a scaled
score s becomes cap tanh(s / cap) before anything else.

In the serving dtype an attention without head mixing, turned values or kept positions, with values as wide as
its keys, runs the kernels of `SoftmaxAttention` (a prompt step reads its own keys and values from the projected rows).

Keys and values live in a paged cache line with separate head sizes.  A step writes its keys and values first
and then (but for those kernels) attends over the line alone, so a prompt, a prompt that continues, a decode step and a layer that reads
the line of another layer (`own_kv=False`: queries only, no key/value tensors of its own) are one code path.
Scores, the mixing, the softmax and the sums are float32 whatever the activations are.
"""
from __future__ import annotations

import torch

from ..cache.cache import KVNeed
from ..weights.loader import TensorSpec
from .base import Mixer, Runtime, StepContext
from .attention import decode_geometry
from .position import RotaryEncoding


class TalkingHeadsAttention(Mixer):
    def __init__(self, hidden: int, n_heads: int, n_kv_heads: int, key_dim: int, value_dim: int, scale: float,
                 position: RotaryEncoding, names: dict[str, str], value_position: RotaryEncoding | None = None,
                 block: int = 0, sink: bool = False, own_kv: bool = True, init_std: float = 0.02, window: int = 0,
                 keep_first: int = 0, values_from_keys: bool = False, unit_norm_eps: float | None = None,
                 gate: str = "element", value_mix: str | None = None, cap: float = 0.0, head_norm_eps: float | None = None):
        if n_heads % n_kv_heads:
            raise ValueError(f"{n_heads} query heads do not divide over {n_kv_heads} key/value heads")
        if gate not in ("head", "element"):
            raise ValueError(f"unknown gate {gate!r} (known: head, element)")
        if values_from_keys and (value_dim != key_dim or value_position is not None or not own_kv):
            raise ValueError("values that are the keys as projected have the keys' size, no turn of their own, and a line of their own")
        if keep_first < 0 or (keep_first and (not window or block)):
            raise ValueError("kept first positions need a window and no blocks")
        self.keep_first = int(keep_first or 0)
        self.values_from_keys = bool(values_from_keys)
        self.unit_norm_eps = None if unit_norm_eps is None else float(unit_norm_eps)
        self.gate = gate
        if value_mix not in (None, "first", "mix") or (value_mix == "mix" and "vmix" not in names):
            raise ValueError(f"value_mix is first or mix (with the checkpoint name of its number, 'vmix'), found {value_mix!r}")
        biases = [b for b in ("q_bias", "k_bias", "v_bias") if b in names]
        if biases and len(biases) != 3:
            raise ValueError("biases stand on all three projections or on none")
        if (biases or value_mix) and (not own_kv or values_from_keys or value_position is not None):
            raise ValueError("biases and mixed values belong to a layer with plain values of its own")
        self.value_mix, self.biased = value_mix, bool(biases)
        if (head_norm_eps is not None) != ("q_norm" in names) or ("q_norm" in names) != ("k_norm" in names):
            raise ValueError("normed heads need head_norm_eps and the checkpoint names of both weights, 'q_norm' and 'k_norm'")
        if head_norm_eps is not None and (biases or not own_kv or values_from_keys):
            raise ValueError("normed heads belong to a layer with keys and values of its own and without biases")
        self.head_norm_eps = None if head_norm_eps is None else float(head_norm_eps)
        self.cap = float(cap or 0.0)
        need = (("q", "k", "o") if values_from_keys else ("q", "k", "v", "o")) if own_kv else ("q", "o")
        for k in need:
            if k not in names:
                raise ValueError(f"attention needs the checkpoint name of its {k!r} projection")
        if value_position is not None and (value_position.rot != value_dim or value_dim % 2):
            raise ValueError("rotated values turn all of their features, in pairs")
        self.hidden, self.n_heads, self.n_kv_heads = hidden, n_heads, n_kv_heads
        self.key_dim, self.value_dim = key_dim, value_dim
        self.scale = float(scale)
        self.block = int(block or 0)
        self.window = int(window or 0)
        if self.window < 0:
            raise ValueError(f"a window holds at least one position, found {window}")
        self.sink = bool(sink) or "sink" in names
        self.own_kv = bool(own_kv)
        self.position, self.value_position = position, value_position
        self.names = dict(names)
        self.init_std = init_std
        self.w_qkv = self.w_o = self.talk = self.bias = self.sink_values = self.wq_norm = self.wk_norm = None
        self.mix_share = 0.0

    def tensor_specs(self):
        H, G, d, dv, W, s, n = self.n_heads, self.n_kv_heads, self.key_dim, self.value_dim, self.hidden, self.init_std, self.names
        specs = {n["q"]: TensorSpec((H * d, W), init_std=s), n["o"]: TensorSpec((W, H * dv), init_std=s)}
        if self.own_kv:
            specs[n["k"]] = TensorSpec((G * d, W), init_std=s)
            if not self.values_from_keys:
                specs[n["v"]] = TensorSpec((G * dv, W), init_std=s)
        if "talk" in n:
            specs[n["talk"]] = TensorSpec((H, H), init_std=H ** -0.5)
        if "g" in n:
            specs[n["g"]] = TensorSpec((H * dv if self.gate == "element" else H, W), init_std=s)
        if self.biased:
            specs.update({n["q_bias"]: TensorSpec((H * d,), init_std=s), n["k_bias"]: TensorSpec((G * d,), init_std=s),
                          n["v_bias"]: TensorSpec((G * dv,), init_std=s)})
        if self.head_norm_eps is not None:
            specs.update({n[k]: TensorSpec((d,), init_std=0.1, init_mean=1.0) for k in ("q_norm", "k_norm")})
        if "sink" in n:
            specs[n["sink"]] = TensorSpec((H,), init_std=1.0)
        if self.value_mix == "mix":
            specs[n["vmix"]] = TensorSpec((), init_std=0.1, init_mean=0.5)
        return specs

    def sub_parts(self):
        return [p for p in (self.position, self.value_position) if p is not None]

    def cache_needs(self):
        return {"kv": KVNeed(self.n_kv_heads, self.key_dim, None, self.value_dim)}

    def prompt_flops(self, n_tokens: int) -> float:
        B = self.block or n_tokens
        full, rest = divmod(n_tokens, B)
        seen = full * (B * (B + 1) // 2) + rest * (rest + 1) // 2         # (query, key) pairs
        if self.window and not self.block:
            w = min(self.window, n_tokens)
            seen = w * (w + 1) // 2 + (n_tokens - w) * w
            far = max(0, n_tokens - w - self.keep_first)          # queries whose window has left all the kept positions behind
            seen += self.keep_first * far + sum(range(1, min(self.keep_first, max(0, n_tokens - w)) + 1)) if self.keep_first else 0
        return seen * 2.0 * self.n_heads * (self.key_dim + self.value_dim + ("talk" in self.names) * self.n_heads)

    def load(self, store, rt: Runtime):
        n = self.names
        gated = ("g",) if "g" in n else ()
        if self.own_kv:
            fused = (("q", "k") if self.values_from_keys else ("q", "k", "v")) + gated
            mats = [store.get(n[x], rt.dtype) for x in fused]
            self.w_qkv = torch.cat(mats, dim=0).contiguous()
            del mats
            store.drop(*(n[x] for x in fused))
        elif gated:
            self.w_qkv = torch.cat([store.get(n["q"], rt.dtype), store.get(n["g"], rt.dtype)], dim=0).contiguous()
            store.drop(n["q"], n["g"])
        else:
            self.w_qkv = store.get(n["q"], rt.dtype).contiguous()
        if self.w_qkv.shape[0] % 8:
            # rows of the step in whole 16-byte pieces (a gate per head may leave any number of columns): zero rows behind the last
            pad = torch.zeros(8 - self.w_qkv.shape[0] % 8, self.w_qkv.shape[1], dtype=self.w_qkv.dtype, device=self.w_qkv.device)
            self.w_qkv = torch.cat([self.w_qkv, pad], dim=0).contiguous()
        self.w_o = store.get(n["o"], rt.dtype).contiguous()
        f32 = lambda k: store.get(n[k]).to(torch.float32)
        self.bias = torch.cat([f32("q_bias"), f32("k_bias"), f32("v_bias")]).contiguous() if self.biased else None
        self.sink_values = f32("sink").contiguous() if "sink" in n else None
        if self.head_norm_eps is not None:
            self.wq_norm, self.wk_norm = f32("q_norm").contiguous(), f32("k_norm").contiguous()
        self.mix_share = float(f32("vmix").reshape(()).item()) if self.value_mix == "mix" else 0.0
        self.talk = store.get(n["talk"]).to(torch.float32).contiguous() if "talk" in n else None

    @property
    def joins(self):
        return "first" if self.own_kv else ""

    def in_weight(self):
        w, self.w_qkv = self.w_qkv, None
        return w

    def out_weight(self):
        w, self.w_o = self.w_o, None
        return w

    def _gate_off(self) -> int:                     # where the gate's logits start in a row
        H, G, d, dv = self.n_heads, self.n_kv_heads, self.key_dim, self.value_dim
        return H * d + ((G * d if self.values_from_keys else G * (d + dv)) if self.own_kv else 0)

    def _gate_run(self) -> int:                     # features that share a gate
        return self.value_dim if self.gate == "head" else 1

    def forward(self, x, ctx: StepContext, line):
        rt, ws = ctx.rt, ctx.ws
        T = ctx.n_tok
        rows = ws.buf("tattn.rows", (T, self.w_qkv.shape[0]), rt.dtype)      # (the product's columns: the gate's, and padding, last)
        rt.linear(x, self.w_qkv, rows)
        return self.finish(rows, 0, ctx, line, ws.buf("mixer.out", (T, self.hidden), rt.dtype))

    def finish(self, rows, col0: int, ctx: StepContext, line, out):
        if col0:
            raise ValueError("an attention's columns are the first of the rows it shares")
        att = self._attend(rows, ctx, line)
        if "g" in self.names:
            ctx.rt.ops.sigmoid_gate(att, rows, self._gate_off(), per=self._gate_run())
        return ctx.rt.linear(att, self.w_o, out)

    def join(self, rows, col0: int, ctx: StepContext, line, z, z0: int, scale: float) -> None:
        if col0:
            raise ValueError("an attention's columns are the first of the rows it shares")
        att = self._attend(rows, ctx, line)
        ctx.rt.ops.gate_place(att, rows if "g" in self.names else None, self._gate_off(), z, z0, scale, per=self._gate_run())

    def _attend(self, rows, ctx: StepContext, line):
        """From the projected rows (q | k | v first) to the heads side by side, [T, H dv]; keys and values are stored."""
        rt, ws, ops = ctx.rt, ctx.ws, ctx.rt.ops
        kv = line["kv"]
        if kv.write != self.own_kv:
            raise ValueError("the schedule lets a layer with keys and values of its own only read a line, or the reverse")
        T, H, G, d, dv = ctx.n_tok, self.n_heads, self.n_kv_heads, self.key_dim, self.value_dim
        inv_v = self.value_position.inv_freq if self.value_position is not None else None
        neighbours = self.position.pairs == "neighbours" and self.position.rot > 0
        if self.values_from_keys or self.unit_norm_eps is not None or neighbours:
            if inv_v is not None or not self.own_kv or self.position.amplitude != 1.0 or self.biased or self.value_mix or self.head_norm_eps is not None:
                raise NotImplementedError("turned or mixed values, biases, a borrowed line or an amplitude together with normed or neighbouring pairs")
            if not self.values_from_keys:
                raise NotImplementedError("normed or neighbouring pairs beside a value projection of its own")
            ops.qk_rotate_norm_store(rows, ctx.tok_pos, ctx.tok_seq, ctx.seq_slot, self.position.inv_freq, self.position.rot,
                                     not neighbours, self.unit_norm_eps is not None, self.unit_norm_eps or 0.0, H, G, d,
                                     kv.k, kv.v if self.values_from_keys else None, kv.table)
        else:
            extras = {}
            if self.biased:
                extras["bias"] = self.bias
            if self.position.amplitude != 1.0:
                extras["amplitude"] = self.position.amplitude
            if self.value_mix == "first":           # (the step's later layers read it: a buffer of its own)
                extras.update(mix=1, v_first=ws.buf("tattn.v_first", (T, G * dv), rt.dtype))
                ctx.shared["first values"] = extras["v_first"]
            elif self.value_mix == "mix":
                extras.update(mix=2, share=self.mix_share, v_first=ctx.shared["first values"])
            if self.head_norm_eps is not None:
                extras.update(q_norm=self.wq_norm, k_norm=self.wk_norm, norm_eps=self.head_norm_eps)
            ops.qkv_rotate_store(rows, ctx.tok_pos, ctx.tok_seq, ctx.seq_slot, self.position.inv_freq, self.position.rot,
                                 inv_v, H, G, d, dv, kv.k if self.own_kv else None, kv.v if self.own_kv else None,
                                 kv.table if self.own_kv else None, store=self.own_kv, **extras)
        att = ws.buf("tattn.ctx", (T, H * dv), rt.dtype)
        if self._plain_heads(rt):
            return self._attend_plain(rows, ctx, kv, att)
        more = {}
        if self.keep_first:
            more["keep_first"] = self.keep_first
        if self.sink_values is not None:
            more["sink_values"] = self.sink_values
        if self.cap:
            more["cap"] = self.cap
        decode = ctx.mode == "decode"
        max_keys, n_chunks, scratch = 0, 1, None
        rows_floats = 0
        if (decode and rt.dtype == torch.bfloat16 and not (self.block and self.window) and self.talk is None and inv_v is None
                and (not self.sink or self.sink_values is not None) and hasattr(ops, "talk_attention_rows_floats")):
            # a decode step in the serving dtype with nothing the kernels that take single rows leave out: keys and
            # values read once, 16 bytes a lane
            max_keys = min(ctx.len_bound, (self.window or self.block) + self.keep_first) if self.window or self.block else ctx.len_bound
            rows_floats = ops.talk_attention_rows_floats(rt.dtype, T, H, G, d, dv, max_keys)
        if rows_floats:
            return ops.talk_attention_rows(rows, ctx.tok_pos, ctx.tok_seq, ctx.seq_slot, kv.k, kv.v, kv.table, None, att, H, G, d, dv,
                                           self.scale, ws.buf("tattn.rows_scratch", (rows_floats,), torch.float32), max_keys,
                                           sink=self.sink, window=self.window or -self.block, **more)
        if decode:
            # a decode row's keys over several CTAs when the rows alone would leave most of the GPU idle: about a
            # CTA an SM in all, none with fewer than 128 keys (the bound on the lengths is the host's)
            max_keys = min(self.block, ctx.len_bound) if self.block else ctx.len_bound
            if self.window:
                max_keys = min(max_keys, self.window + self.keep_first)
            n_chunks = max(1, min(rt.sm_count // max(T, 1), -(-max_keys // 128), 64))
            n = ops.talk_attention_scratch_floats(T, n_chunks, H, dv)
            scratch = ws.buf("tattn.partial", (n,), torch.float32) if n else None
        return ops.talk_attention(rows, ctx.tok_pos, ctx.tok_seq, ctx.seq_slot, kv.k, kv.v, kv.table, self.talk, inv_v, att,
                                  H, G, d, dv, self.scale, self.block, self.sink, one_row=decode, max_keys=max_keys,
                                  n_chunks=n_chunks, scratch=scratch, window=self.window, **more)

    def _plain_heads(self, rt) -> bool:
        """Whether the kernels of whole heads (one head a CTA, keys and values of one size) take this attention."""
        return (self.talk is None and not (self.block and self.window) and self.value_position is None and not self.keep_first and self.own_kv
                and not self.values_from_keys and (not self.sink or self.sink_values is not None) and hasattr(rt.ops, "attn_rows_sizes")
                and rt.ops.attn_rows_sizes(rt.dtype, self.n_heads, self.n_kv_heads, self.key_dim, self.value_dim))

    def _attend_plain(self, rows, ctx: StepContext, kv, att):
        rt, ws, ops = ctx.rt, ctx.ws, ctx.rt.ops
        H, G, d = self.n_heads, self.n_kv_heads, self.key_dim
        seen = self.window or -self.block                      # (a negative window: chunks of that many positions)
        if ctx.mode == "decode":
            chunk, max_chunks = decode_geometry(ctx, rt.sm_count, d, G, abs(seen))
            scratch = ws.buf("attn.partial", (ops.attn_decode_scratch_floats(ctx.n_seq, H, d, max_chunks),), torch.float32)
            return ops.attn_decode_rows(rows, kv.k, kv.v, kv.table, ctx.seq_slot, ctx.seq_end, scratch, att, H, G, d, self.scale,
                                        seen, chunk, max_chunks, cap=self.cap, sinks=self.sink_values)
        n_scratch = ops.attn_prefill_scratch_floats(ctx.n_tok, ctx.n_seq, H, d, rt.dtype)
        scratch = ws.buf("attn.prefill_partial", (n_scratch,), torch.float32) if n_scratch else None
        before = dict(seq_start=ctx.seq_start, seq_slot=ctx.seq_slot, kpool=kv.k, vpool=kv.v, page_table=kv.table) if ctx.extends else {}
        return ops.attn_prefill_rows(rows, ctx.seq_first_row, ctx.seq_end, att, H, G, d, self.scale, seen, cap=self.cap,
                                     sinks=self.sink_values, scratch=scratch, host_lens=ctx.step_lens, **before)
