"""Gated delta rule: a recurrent mixer whose state is a matrix per head that every token corrects towards its value.

With y the mixer's input, H heads over G query/key heads (head h uses h // (H/G)), d key channels, dv value channels:

    q, k, v = silu(conv(W_q y)), silu(conv(W_k y)), silu(conv(W_v y))      conv: causal, per channel, `taps` taps, no bias
    q, k      <- x / sqrt(sum(x^2) + 1e-6) per head; q also times q_scale
    beta = sigmoid(W_b y),   g = exp(-exp(A_log) softplus(W_a y + dt_bias))      one of each per head
    S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q               S starts at zero, lives in the cache, float32

then each head's o is RMS-normed over its dv channels (one weight vector for all heads), the heads side by side are multiplied
by silu(W_g y) and projected by W_o.  The projections of y are one product over the rows q | k | v | g | b | a concatenated at
load; the three convolutions are one over the channels q | k | v.  From the convolved values on everything is float32 whatever
the activations are: unit norms, gates, decays, the state and o.

A cache line holds two fixed-size parts: the state (S^T: [heads, dv, d]) and the last taps - 1 inputs of the convolution; a
step loads them, runs its tokens in order and writes them back.  Prompts and prompts that continue run the recurrence four
tokens at a time; a decode step runs one kernel that also norms and gates the output.  Sequences without a slot (padding)
start from zero and store nothing.
"""
from __future__ import annotations

import torch

from ..cache.cache import StateNeed
from ..weights.loader import TensorSpec
from .base import Mixer, Runtime, StepContext


class GatedDeltaRule(Mixer):
    NAMES = ("q", "k", "v", "g", "b", "a", "q_conv", "k_conv", "v_conv", "A_log", "dt_bias", "norm", "o")

    def __init__(self, hidden: int, n_heads: int, n_key_heads: int, key_dim: int, value_dim: int, taps: int, norm_eps: float,
                 names: dict[str, str], q_scale: float | None = None, init_std: float = 0.02):
        for k in self.NAMES:
            if k not in names:
                raise ValueError(f"the gated delta rule needs the checkpoint name of its {k!r} tensor")
        if n_heads % n_key_heads:
            raise ValueError(f"{n_heads} heads do not divide over {n_key_heads} query/key heads")
        if key_dim > 256:
            raise ValueError(f"the recurrence kernels take up to 256 key channels a head, found {key_dim}")
        if not 1 <= taps <= 16:
            raise ValueError(f"the convolution kernel takes 1 to 16 taps, found {taps}")
        self.hidden, self.n_heads, self.n_key_heads = hidden, n_heads, n_key_heads
        self.key_dim, self.value_dim, self.taps = key_dim, value_dim, int(taps)
        self.norm_eps = float(norm_eps)
        self.q_scale = float(q_scale) if q_scale is not None else key_dim ** -0.5
        self.channels = 2 * n_key_heads * key_dim + n_heads * value_dim            # q | k | v
        self.names = dict(names)
        self.init_std = init_std
        self.w_in = self.w_conv = self.decay = self.dt_bias = self.w_norm = self.w_o = None

    def tensor_specs(self):
        H, G, d, dv, W, s, n = self.n_heads, self.n_key_heads, self.key_dim, self.value_dim, self.hidden, self.init_std, self.names
        specs = {n["q"]: TensorSpec((G * d, W), init_std=s), n["k"]: TensorSpec((G * d, W), init_std=s),
                 n["v"]: TensorSpec((H * dv, W), init_std=s), n["g"]: TensorSpec((H * dv, W), init_std=s),
                 n["b"]: TensorSpec((H, W), init_std=s), n["a"]: TensorSpec((H, W), init_std=s),
                 n["A_log"]: TensorSpec((H,), init_std=1.0, init_mean=-2.0), n["dt_bias"]: TensorSpec((H,), init_std=1.0, init_mean=-2.0),
                 n["norm"]: TensorSpec((dv,), init_std=0.1, init_mean=1.0), n["o"]: TensorSpec((W, H * dv), init_std=s)}
        for key, rows in (("q_conv", G * d), ("k_conv", G * d), ("v_conv", H * dv)):
            specs[n[key]] = TensorSpec((rows, self.taps), init_std=self.taps ** -0.5)
        return specs

    def cache_needs(self):
        return {"state": StateNeed((self.n_heads, self.value_dim, self.key_dim), torch.float32),             # S^T per head
                "conv": StateNeed((max(self.taps - 1, 1), self.channels), torch.float32)}

    def prompt_flops(self, n_tokens: int) -> float:
        # two products with the state, its decay and its update; the filter
        return n_tokens * (7.0 * self.n_heads * self.key_dim * self.value_dim + 2.0 * self.channels * self.taps)

    def load(self, store, rt: Runtime):
        n = self.names
        order = ("q", "k", "v", "g", "b", "a")
        mats = [store.get(n[k], rt.dtype) for k in order]
        pad = -sum(m.shape[0] for m in mats) % 8           # rows of the step in whole 16-byte pieces: zero rows behind the last
        if pad:
            mats.append(torch.zeros(pad, self.hidden, dtype=rt.dtype, device=mats[0].device))
        self.w_in = torch.cat(mats, dim=0).contiguous()
        del mats
        store.drop(*(n[k] for k in order))
        f32 = lambda k: store.get(n[k]).to(torch.float32)
        self.w_conv = torch.cat([f32("q_conv"), f32("k_conv"), f32("v_conv")], dim=0).contiguous()
        self.decay = (-torch.exp(f32("A_log"))).contiguous()
        self.dt_bias = f32("dt_bias").contiguous()
        self.w_norm = f32("norm").contiguous()
        self.w_o = store.get(n["o"], rt.dtype).contiguous()

    joins = "any"

    def in_weight(self):
        w, self.w_in = self.w_in, None
        return w

    def out_weight(self):
        w, self.w_o = self.w_o, None
        return w

    def forward(self, x, ctx: StepContext, line):
        rows = ctx.rt.linear(x, self.w_in, ctx.ws.buf("delta.rows", (ctx.n_tok, self.w_in.shape[0]), ctx.rt.dtype))
        return self.finish(rows, 0, ctx, line, ctx.ws.buf("mixer.out", (ctx.n_tok, self.hidden), ctx.rt.dtype))

    def finish(self, rows, col0: int, ctx: StepContext, line, out):
        return ctx.rt.linear(self._heads(rows, col0, ctx, line), self.w_o, out)

    def join(self, rows, col0: int, ctx: StepContext, line, z, z0: int, scale: float) -> None:
        ctx.rt.ops.gate_place(self._heads(rows, col0, ctx, line), None, 0, z, z0, scale)

    def _heads(self, rows, col0: int, ctx: StepContext, line):
        """From its columns of the projected rows to the normed and gated heads side by side, [T, H dv]."""
        rt, ws, ops = ctx.rt, ctx.ws, ctx.rt.ops
        st, cv = line["state"], line["conv"]
        if not st.write:
            raise ValueError("a recurrent state has one writer: a delta-rule layer cannot read another's line")
        T, H, G, d, dv, C = ctx.n_tok, self.n_heads, self.n_key_heads, self.key_dim, self.value_dim, self.channels
        g_off = col0 + C
        b_off, a_off = g_off + H * dv, g_off + H * dv + H
        one = ctx.mode == "decode"
        x = ws.buf("delta.x", (T, C), rt.dtype)
        ops.causal_conv_silu(rows, col0, C, self.w_conv, None, cv.data, ctx.tok_seq, ctx.seq_slot, ctx.seq_first_row, ctx.seq_start,
                             ctx.seq_end, ctx.n_seq, x, one_token=one)
        y = ws.buf("delta.y", (T, H * dv), rt.dtype)
        offs = (0, G * d, 2 * G * d)
        if one:
            return ops.delta_step(x, *offs, rows, a_off, b_off, g_off, self.decay, self.dt_bias, self.q_scale, self.w_norm,
                                  self.norm_eps, ctx.tok_seq, ctx.seq_slot, st.data, y, H, G, d, dv)
        o = ws.buf("delta.o", (T, H * dv), torch.float32)
        ops.delta_scan(x, *offs, rows, a_off, b_off, self.decay, self.dt_bias, self.q_scale, ctx.tok_pos, ctx.tok_seq, ctx.seq_slot,
                       ctx.seq_first_row, ctx.seq_start, ctx.seq_end, st.data, o, ctx.n_seq, H, G, d, dv,
                       ws.buf("delta.coef", (T, H, ops.DELTA_COEF), torch.float32))
        return ops.head_norm_gate(o, rows, g_off, self.w_norm, self.norm_eps, y, H, dv)
