"""Plain, slow Mugedra: whole sequences, no cache, one function per mechanism.

It is the oracle of the Mugedra tests and shares no code with the package under
test (the container reader is the other oracle's).  Everything runs in float64
torch operations.

The design, in this file's notation.  r is the residual stream [T, width], y a sublayer's input.

* embedding:     r = E[token] = r0
* layer:         r += ls1 * mixer(N1(r));  r += ls2 * ff(N2(r))      (the second only with a feed-forward; * per feature)
* norm:          N(r) = (r - mean) / sqrt(mean((r - mean)^2) + eps) * w
* loop:          a run of layers is passed several times; r += r0 before every pass but the first
* mixer:         out = (rms(left(y)) * w_l + rms(right(y)) * w_r) / 2,   rms(x) = x / sqrt(mean(x^2) + eps)
   left:         grouped softmax attention: q and k normed per head (rms, one weight for all heads), then turned on their
                 first rot.dims features (pairs i, i + dims/2; frequencies blended between f and f / factor over a ramp, sine
                 and cosine times 0.1 ln(factor) + 1); s = cap tanh(scale q.k / cap); a key is seen by the queries behind
                 it in its own chunk of `size` positions; the heads times sigmoid(W_g y); W_o
   right:        q, k, v = silu(conv(W y)); q and k to unit vectors per head (q also times dim^-1/2);
                 beta = sigmoid(W_b y), a = exp(-exp(A_log) softplus(W_a y + dt_bias)), one each per head;
                 S <- a S;  S <- S + k (beta (v - S^T k))^T;  o = S^T q;  W_o (rms(o) * w * silu(W_g y))
* feed-forward:  moe: s = sigmoid(W_router y), the `top` largest are chosen; sum over them of expert(s_e y),
                 expert(u) = W_down (silu(W_gate u) * (W_up u))
* output:        final norm, head
"""
from __future__ import annotations

import math

import torch

from .gemma2_plain import load_folder  # noqa: F401  (the folder reader: config dict and float64 tensors)

F = torch.float64


def layer_norm(x, weight, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * weight


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def softplus(x):
    return torch.logaddexp(x, torch.zeros_like(x))


def silu(x):
    return x * torch.sigmoid(x)


# ---------------------------------------------------------------------------
# attention
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


def attend(q, k, v, scale, cap=0.0, chunk=0):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: causal softmax attention inside chunks of positions (chunk 0: everywhere),
    capped scores (cap 0: the scores themselves)."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    at = torch.arange(T)
    seen = at[None, :] <= at[:, None]
    if chunk:
        seen &= (at[None, :] // chunk) == (at[:, None] // chunk)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        out[:, h] = torch.softmax(s.masked_fill(~seen, -math.inf), dim=1) @ v[:, h // rep]
    return out


def gated_attention(y, w, pre, m, eps):
    T = y.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    freq, amp = frequencies(m["rot"]) if m.get("rot") else (torch.zeros(0, dtype=F), 1.0)
    q = turn(rms_norm((y @ w[pre + "q"].T).view(T, H, d), w[pre + "q.norm"], eps), pos, freq, amp)
    k = turn(rms_norm((y @ w[pre + "k"].T).view(T, G, d), w[pre + "k.norm"], eps), pos, freq, amp)
    v = (y @ w[pre + "v"].T).view(T, G, dv)
    o = attend(q, k, v, m["scale"], m.get("softcap") or 0.0, m["mask"]["size"] if m.get("mask") else 0).reshape(T, H * dv)
    return (o * torch.sigmoid(y @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---------------------------------------------------------------------------
# the gated delta rule
# ---------------------------------------------------------------------------

def causal_conv(x, kernel):
    """x [T, C], kernel [C, taps]: out[t, c] = sum_j kernel[c, taps - 1 - j] x[t - j, c], zeros before t = 0."""
    T, C = x.shape
    taps = kernel.shape[1]
    out = torch.zeros(T, C, dtype=F)
    for j in range(min(taps, T)):
        out[j:] += kernel[:, taps - 1 - j] * x[:T - j]
    return out


def decay(z, A_log, dt_bias):
    return torch.exp(-torch.exp(A_log) * softplus(z + dt_bias))


def delta_rule(q, k, v, g, beta):
    """q, k [T, H, d], v [T, H, dv], g, beta [T, H]: the read-outs o [T, H, dv] of a state that starts at zero."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def delta_mixer(y, w, pre, m, eps):
    T = y.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(y @ w[pre + n].T, w[pre + n + ".conv"])) for n in "qkv")
    rep = H // G
    q = (unit(q.view(T, G, d)) * d ** -0.5).repeat_interleave(rep, dim=1)
    k = unit(k.view(T, G, d)).repeat_interleave(rep, dim=1)
    o = delta_rule(q, k, v.view(T, H, dv), decay(y @ w[pre + "a"].T, w[pre + "A_log"], w[pre + "dt_bias"]),
                   torch.sigmoid(y @ w[pre + "b"].T))
    o = rms_norm(o, w[pre + "norm"], eps).reshape(T, H * dv) * silu(y @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


def parallel_mixer(y, w, pre, m, eps):
    left = gated_attention(y, w, pre + "left.", m["left"], eps)
    right = delta_mixer(y, w, pre + "right.", m["right"], eps)
    return 0.5 * (rms_norm(left, w[pre + "left.out"], eps) + rms_norm(right, w[pre + "right.out"], eps))


# ---------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------

def expert(u, w, pre):
    return (silu(u @ w[pre + "gate"].T) * (u @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(z, top):
    """z [T, E] router logits: (chosen experts [T, top], their weights)."""
    s = torch.sigmoid(z)
    idx = s.topk(top, dim=-1).indices
    return idx, s.gather(1, idx)


def moe_ff(y, w, pre, mlp):
    idx, wts = route(y @ w[pre + "router"].T, mlp["router"]["top"])
    out = torch.zeros_like(y)
    for t in range(y.shape[0]):
        for e, a in zip(idx[t].tolist(), wts[t]):
            out[t] += expert(a * y[t:t + 1], w, f"{pre}e{e}.")[0]
    return out


# ---------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------

def layer_order(n_layers, loop):
    """[(layer, whether the embedding output is added before it)] in the order the layers run."""
    if not loop:
        return [(i, False) for i in range(n_layers)]
    a, b = loop["start"], loop["stop"]
    order = [(i, False) for i in range(a)]
    for p in range(loop["times"]):
        order += [(i, p > 0 and i == a) for i in range(a, b)]
    return order + [(i, False) for i in range(b, n_layers)]


def forward(cfg, w, tokens, after=None):
    """float64 logits [T, vocab] of a whole sequence from position 0; `after` (a list) gets the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    r = w["embed"][torch.as_tensor(tokens)]
    r0 = r
    for i, again in layer_order(len(cfg["layers"]), cfg.get("loop")):
        layer, p = cfg["layers"][i], f"l{i}."
        if layer["type"] != "parallel":
            raise ValueError(layer["type"])
        if again:
            r = r + r0
        r = r + w[p + "ls1"] * parallel_mixer(layer_norm(r, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            r = r + w[p + "ls2"] * moe_ff(layer_norm(r, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"])
        if after is not None:
            after.append(r.clone())
    return layer_norm(r, w["final.norm"], eps) @ w["head"].T
