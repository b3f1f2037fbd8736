"""Plain, slow Larulorn: whole sequences, no cache, one function per mechanism.

It is the oracle of the Larulorn tests and shares no code with the package under
test (the container reader is the other oracle's).  Everything runs in float64
torch operations.

The design, in this file's notation.  r is the residual stream [T, width], y a sublayer's input.

* embedding:     r = E[token]
* layer:         r += N1b(mixer(N1(r)));  r += N2b(ff(N2(r)))        (the second line only with a feed-forward)
* norm:          N(r) = r / sqrt(mean(r^2) + eps) * w
* 'attention':   q, k, v = W y + b; q and k turned on their first rot.dims features (pairs i, i + dims/2), frequencies
                 blended between f and f / factor over a ramp, sine and cosine times 0.1 ln(factor) + 1; causal softmax
                 whose denominator also holds exp(sink_h); values, in layers that mix them: v <- (1 - m) v + m v0 with v0 the
                 values of the first such layer; W_o
* 'parallel':    out = s_l left(y) + s_r right(y) with
   left:         grouped causal softmax attention, plain turned positions, the heads times sigmoid(W_g y), W_o
   right:        u = conv(W_x y + b_x);  ri, ii = sigmoid of a square product per block of u's channels;
                 log a = -8 ri softplus(lam);  S_t = a S_{t-1} + sqrt(1 - a^2) ii u;  W_o (S * gelu_tanh(W_y y + b_y))
* feed-forward:  dense: g = min(W_gate y, limit), u = clamp(W_up y, +-limit), W_down (g sigmoid(1.702 g) (u + 1));
                 moe: softmax router over groups of experts, experts W_down relu(W_up y)^2, a shared one added
* output:        final norm, head, times logit_scale
"""
from __future__ import annotations

import math

import torch

from .gemma2_plain import load_folder  # noqa: F401  (the folder reader: config dict and float64 tensors)

F = torch.float64


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def softplus(x):
    return torch.logaddexp(x, torch.zeros_like(x))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------------------
# positions
# ---------------------------------------------------------------------------

def frequencies(rot):
    """(frequencies, amplitude): base^(-2i/dims), and with rot.scaling the blend over the ramp."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc or not dims:
        return torch.tensor(f, dtype=F), 1.0
    factor, original = sc["factor"], sc["original"]

    def where(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / factor * r + v * (1.0 - r))
    return torch.tensor(out, dtype=F), 0.1 * math.log(factor) + 1.0


def turn(x, pos, freq, amplitude=1.0):
    """x [T, heads, n]: the first 2 len(freq) features turned by pos * freq, pairs (i, i + len(freq))."""
    h = freq.numel()
    if h == 0:
        return x
    ang = pos.to(F)[:, None] * freq[None, :]
    c, s = amplitude * torch.cos(ang)[:, None, :], amplitude * torch.sin(ang)[:, None, :]
    a, b = x[..., :h], x[..., h:2 * h]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., 2 * h:]], dim=-1)


# ---------------------------------------------------------------------------
# mixers
# ---------------------------------------------------------------------------

def attend(q, k, v, scale, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: causal softmax attention; sink [H]: exp(sink_h) joins head h's denominator."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    seen = torch.tril(torch.ones(T, T, dtype=torch.bool))
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * scale
        s = s.masked_fill(~seen, -math.inf)
        top = s.max(dim=1, keepdim=True).values
        if sink is not None:
            top = torch.maximum(top, sink[h].expand_as(top))
        e = torch.exp(s - top)
        den = e.sum(1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - top)
        out[:, h] = (e / den) @ v[:, h // rep]
    return out


def mix_values(v, first, m):
    return (1.0 - m) * v + m * first


def sink_attention(y, w, pre, m, first_values):
    """Returns (output, the values as projected, which later layers mix in)."""
    T = y.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    freq, amp = frequencies(m["rot"]) if m.get("rot") else (torch.zeros(0, dtype=F), 1.0)
    q = turn((y @ w[pre + "q"].T + w[pre + "q.b"]).view(T, H, d), pos, freq, amp)
    k = turn((y @ w[pre + "k"].T + w[pre + "k.b"]).view(T, G, d), pos, freq, amp)
    v = (y @ w[pre + "v"].T + w[pre + "v.b"]).view(T, G, dv)
    own = v
    if m.get("v_mix") and first_values is not None:
        v = mix_values(v, first_values, w[pre + "vmix"].reshape(()))
    o = attend(q, k, v, m["scale"], w[pre + "sink"])
    return o.reshape(T, H * dv) @ w[pre + "o"].T, own


def gated_attention(y, w, pre, m):
    T = y.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    freq, amp = frequencies(m["rot"]) if m.get("rot") else (torch.zeros(0, dtype=F), 1.0)
    q = turn((y @ w[pre + "q"].T).view(T, H, d), pos, freq, amp)
    k = turn((y @ w[pre + "k"].T).view(T, G, d), pos, freq, amp)
    v = (y @ w[pre + "v"].T).view(T, G, dv)
    o = attend(q, k, v, m["scale"]).reshape(T, H * dv)
    return (o * torch.sigmoid(y @ w[pre + "g"].T)) @ w[pre + "o"].T


def causal_conv(x, kernel, bias):
    """x [T, C], kernel [C, taps]: out[t, c] = bias[c] + sum_j kernel[c, taps - 1 - j] x[t - j, c], zeros before t = 0."""
    T, C = x.shape
    taps = kernel.shape[1]
    out = bias.expand(T, C).clone()
    for j in range(min(taps, T)):
        out[j:] += kernel[:, taps - 1 - j] * x[:T - j]
    return out


def block_gate(u, mats, bias):
    """sigmoid(mats[b] u_b + bias[b]) over equal runs u_b of u's channels; mats [blocks, n, n]."""
    T = u.shape[0]
    n_b, n, _ = mats.shape
    z = torch.einsum("tbi,boi->tbo", u.view(T, n_b, n), mats) + bias[None]
    return torch.sigmoid(z).reshape(T, n_b * n)


def linear_recurrence(u, gate_r, gate_i, lam):
    """S_t = a S_{t-1} + sqrt(1 - a^2) i u with log a = -8 r softplus(lam), S before the first token 0; all S_t."""
    S = torch.zeros(u.shape[1], dtype=F)
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        a = torch.exp(-8.0 * gate_r[t] * softplus(lam))
        S = a * S + torch.sqrt(1.0 - a * a) * gate_i[t] * u[t]
        out[t] = S
    return out


def recurrent_block(y, w, pre, m):
    branch = gelu_tanh(y @ w[pre + "y"].T + w[pre + "y.b"])
    u = causal_conv(y @ w[pre + "x"].T + w[pre + "x.b"], w[pre + "conv"], w[pre + "conv.b"])
    S = linear_recurrence(u, block_gate(u, w[pre + "ra"], w[pre + "ra.b"]), block_gate(u, w[pre + "ri"], w[pre + "ri.b"]),
                          w[pre + "lam"])
    return (S * branch) @ w[pre + "o"].T


def parallel_mixer(y, w, pre, m):
    return m["left_scale"] * gated_attention(y, w, pre + "left.", m["left"]) \
        + m["right_scale"] * recurrent_block(y, w, pre + "right.", m["right"])


# ---------------------------------------------------------------------------
# feed-forwards
# ---------------------------------------------------------------------------

def clamped_gate(y, w, pre, limit):
    g = torch.clamp(y @ w[pre + "gate"].T, max=limit)
    u = torch.clamp(y @ w[pre + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[pre + "down"].T


def expert(y, w, pre):
    return torch.relu(y @ w[pre + "up"].T) ** 2 @ w[pre + "down"].T


def route(z, top, groups=None):
    """z [T, E] router logits: (chosen experts [T, top], their weights)."""
    T, E = z.shape
    s = torch.softmax(z, dim=-1)
    running = s.clone()
    if groups:
        per = E // groups["count"]
        best = s.view(T, groups["count"], per).max(dim=-1).values.topk(groups["keep"], dim=-1).indices
        for t in range(T):
            for g in range(groups["count"]):
                if g not in best[t].tolist():
                    running[t, g * per:(g + 1) * per] = -1.0
    idx = running.topk(top, dim=-1).indices
    chosen = s.gather(1, idx)
    return idx, chosen / (chosen.sum(-1, keepdim=True) + 1e-20)


def moe_ff(y, w, pre, mlp):
    idx, wts = route(y @ w[pre + "router"].T, mlp["router"]["top"], mlp["router"].get("groups"))
    out = torch.zeros_like(y)
    for t in range(y.shape[0]):
        for e, a in zip(idx[t].tolist(), wts[t]):
            out[t] += a * expert(y[t:t + 1], w, f"{pre}e{e}.")[0]
    if mlp.get("shared"):
        out = out + expert(y, w, pre + "shared.")
    return out


# ---------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------

def forward(cfg, w, tokens, after=None):
    """float64 logits [T, vocab] of a whole sequence from position 0; `after` (a list) gets the stream after every layer."""
    eps = cfg["norm"]["eps"]
    r = w["embed"][torch.as_tensor(tokens)]
    first_values = None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = rms_norm(r, w[p + "norm1"], eps)
        if layer["type"] == "attention":
            o, values = sink_attention(y, w, p + "mix.", layer["mixer"], first_values)
            if layer["mixer"].get("v_mix") and first_values is None:
                first_values = values
        elif layer["type"] == "parallel":
            o = parallel_mixer(y, w, p + "mix.", layer["mixer"])
        else:
            raise ValueError(layer["type"])
        r = r + rms_norm(o, w[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp:
            y = rms_norm(r, w[p + "norm2"], eps)
            o = clamped_gate(y, w, p + "mlp.", mlp["limit"]) if mlp["kind"] == "dense" else moe_ff(y, w, p + "mlp.", mlp)
            r = r + rms_norm(o, w[p + "norm2b"], eps)
        if after is not None:
            after.append(r.clone())
    return rms_norm(r, w["final.norm"], eps) @ w["head"].T * cfg.get("logit_scale", 1.0)
