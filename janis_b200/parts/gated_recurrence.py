"""The recurrent block with a real-gated linear recurrent unit (Griffin's), as a mixer: one number of state per channel.

With y the mixer's input and C channels in equal blocks of n:

    u  = conv(W_x y + b_x)                                a causal convolution per channel, with its own bias, no activation
    r  = sigmoid(A_r[b] u_b + a_r[b]),  i = sigmoid(A_i[b] u_b + a_i[b])      block b's channels: square products
    log a = -rate r softplus(lam)
    S <- a S + sqrt(1 - a^2) i u                          S starts at zero, for the first token too
    out = W_o (S * gelu_tanh(W_y y + b_y))

The two projections are one product over the rows W_y | W_x.  The gates' logits are float32 results of a product per
block (of bfloat16 operands in the serving path); they, the decays, the input's factor and S are float32 whatever the
activations are.  The cache line holds S [C] in float32 and the convolution's last taps - 1 inputs (with b_x, so that they
are zero before the sequence's start); a step loads them, runs its tokens in order and writes them back, so a prompt, a
prompt that continues and a decode step leave the same state.  In a decode step the gates' products, the recurrence and
the branch's activation are one kernel.
"""
from __future__ import annotations

import torch

from ..cache.cache import StateNeed
from ..weights.loader import TensorSpec
from .base import Mixer, Runtime, StepContext
from .state_space import _conv_need


class GatedRecurrenceMixer(Mixer):
    NAMES = ("y", "y_bias", "x", "x_bias", "conv", "conv_bias", "ra", "ra_bias", "ri", "ri_bias", "lam", "o")
    joins = "any"

    def __init__(self, hidden: int, width: int, blocks: int, taps: int, names: dict[str, str], rate: float = 8.0,
                 init_std: float = 0.02):
        for k in self.NAMES:
            if k not in names:
                raise ValueError(f"the gated recurrence needs the checkpoint name of its {k!r} tensor")
        if width % blocks:
            raise ValueError(f"{width} channels do not divide into {blocks} blocks")
        if width // blocks > 1536:
            raise ValueError(f"the recurrence kernel takes blocks of up to 1536 channels, found {width // blocks}")
        if not 1 <= taps <= 16:
            raise ValueError(f"the convolution kernel takes 1 to 16 taps, found {taps}")
        self.hidden, self.width, self.blocks, self.taps, self.rate = hidden, width, blocks, taps, float(rate)
        self.names = dict(names)
        self.init_std = init_std
        self.w_in = self.w_conv = self.b_conv = self.b_x = self.b_y = None
        self.w_gates = self.b_r = self.b_i = self.decay = self.w_o = None

    def tensor_specs(self):
        W, C, B, s, n = self.hidden, self.width, self.blocks, self.init_std, self.names
        m = C // B
        return {n["y"]: TensorSpec((C, W), init_std=s), n["y_bias"]: TensorSpec((C,), init_std=0.1),
                n["x"]: TensorSpec((C, W), init_std=s), n["x_bias"]: TensorSpec((C,), init_std=0.1),
                n["conv"]: TensorSpec((C, self.taps), init_std=0.3), n["conv_bias"]: TensorSpec((C,), init_std=0.1),
                n["ra"]: TensorSpec((B, m, m), init_std=m ** -0.5), n["ra_bias"]: TensorSpec((B, m), init_std=1.0),
                n["ri"]: TensorSpec((B, m, m), init_std=m ** -0.5), n["ri_bias"]: TensorSpec((B, m), init_std=1.0),
                n["lam"]: TensorSpec((C,), init_std=1.5, init_mean=-4.0), n["o"]: TensorSpec((W, C), init_std=s)}

    def cache_needs(self):
        return {"state": StateNeed((self.width,), torch.float32), "conv": _conv_need(self.taps, self.width)}

    def prompt_flops(self, n_tokens: int) -> float:
        return (4.0 * self.width // self.blocks + 2.0 * self.taps + 6.0) * self.width * n_tokens     # gates' products, filter, recurrence

    def load(self, store, rt: Runtime):
        n, C = self.names, self.width
        f32 = lambda k: store.get(n[k]).to(torch.float32).contiguous()
        self.w_in = torch.cat([store.get(n["y"], rt.dtype), store.get(n["x"], rt.dtype)], dim=0).contiguous()
        store.drop(n["y"], n["x"])
        self.b_y, self.b_x = f32("y_bias"), f32("x_bias")
        self.w_conv, self.b_conv = f32("conv"), f32("conv_bias")
        self.w_gates = torch.cat([store.get(n["ra"], rt.dtype), store.get(n["ri"], rt.dtype)], dim=1).contiguous()    # [B, 2 n, n]
        store.drop(n["ra"], n["ri"])
        self.b_r, self.b_i = f32("ra_bias").reshape(C), f32("ri_bias").reshape(C)
        lam = store.get(n["lam"]).to(torch.float64)
        self.decay = (-self.rate * torch.logaddexp(lam, torch.zeros_like(lam))).to(torch.float32).contiguous()
        self.w_o = store.get(n["o"], rt.dtype).contiguous()

    def in_weight(self):
        w, self.w_in = self.w_in, None
        return w

    def out_weight(self):
        w, self.w_o = self.w_o, None
        return w

    def forward(self, x, ctx: StepContext, line):
        rt, ws = ctx.rt, ctx.ws
        T, C = ctx.n_tok, self.width
        rows = rt.linear(x, self.w_in, ws.buf("rec.in", (T, 2 * C), rt.dtype))
        z = ws.buf("rec.z", (T, C), rt.dtype)
        self.join(rows, 0, ctx, line, z, 0, 1.0)
        return rt.linear(z, self.w_o, ws.buf("mixer.out", (T, self.hidden), rt.dtype))

    def join(self, rows, col0: int, ctx: StepContext, line, z, z0: int, scale: float) -> None:
        rt, ws, ops = ctx.rt, ctx.ws, ctx.rt.ops
        st, cv = line["state"], line["conv"]
        if not st.write:
            raise ValueError("a recurrent state has one writer: a recurrence layer cannot read another's line")
        T, C, B = ctx.n_tok, self.width, self.blocks
        m = C // B
        decode = ctx.mode == "decode"
        u = ws.buf("rec.u", (T, C), rt.dtype)
        ops.causal_conv_silu(rows, col0 + C, C, self.w_conv, self.b_conv, cv.data, ctx.tok_seq, ctx.seq_slot, ctx.seq_first_row,
                             ctx.seq_start, ctx.seq_end, ctx.n_seq, u, one_token=decode, act=False, in_bias=self.b_x)
        if decode:
            ops.gated_recurrence_rows(u, self.w_gates, self.b_r, self.b_i, self.decay, rows, col0, self.b_y, ctx.tok_seq,
                                      ctx.seq_slot, st.data, z, z0, scale)
            return
        gates = ws.buf("rec.gates", (T, B, 2 * m), torch.float32)
        ops.head_linear(u, m, 0, self.w_gates, gates.view(T, 2 * C), 2 * m, 0)
        ops.gated_recurrence_scan(u, gates, m, self.b_r, self.b_i, self.decay, rows, col0, self.b_y, ctx.seq_slot,
                                  ctx.seq_first_row, ctx.seq_start, ctx.seq_end, ctx.n_seq, st.data, z, z0, scale)
