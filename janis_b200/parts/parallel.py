"""Mixers side by side: several mixers read the same input and their outputs are averaged, or added with constant
weights.

    out = (1 / n) sum_i  rms(mixer_i(y)) * w_i          rms(x) = x / sqrt(mean(x^2) + eps) over the model width
    out = sum_i scale_i mixer_i(y)                      with `scales`

In the first form each branch's output is normed with a weight vector of its own (plain, no offset) before the mean, so
that branches of different scale count alike.  The norms and the sum are float32; the result is handed to the block
as float32 and enters the residual sum unrounded.

With `deferred` the first form hands the block its branches as they are (`NormedBranches`, at most two) and leaves norms
and mean to the kernel that adds them to the stream; the branches then share their first product too.

In the second form the branches share their products (`Mixer.join`): one product of y gives every branch its columns,
and the branches' features, each times its constant, stand side by side as the input of one output product over the
concatenated output matrices, which is the weighted sum.

The branches keep what they need in the same cache line, under their own names (`left.kv`, `right.state`, ...):
the line a branch sees holds its parts alone.
"""
from __future__ import annotations

import torch

from ..cache.cache import CacheLine
from ..weights.loader import TensorSpec
from .base import Mixer, Runtime, StepContext
from .norm import NormedBranches


class ParallelMixers(Mixer):
    def __init__(self, hidden: int, branches: dict[str, Mixer], out_norm_names: dict[str, str] | None = None, eps: float = 0.0,
                 init_std: float = 0.1, scales: dict[str, float] | None = None, deferred: bool = False):
        if not branches:
            raise ValueError("parallel mixers need at least one branch")
        if (scales is None) == (out_norm_names is None):
            raise ValueError("parallel mixers are normed and averaged, or added with a constant each")
        if deferred and (scales is not None or len(branches) > 2):
            raise ValueError("one or two branches that are normed and averaged can be left to the block")
        self.deferred = bool(deferred)
        if scales is not None or deferred:
            for at, (k, m) in enumerate(branches.items()):
                if scales is not None and k not in scales:
                    raise ValueError(f"branch {k!r} needs its constant")
                if m.joins != "any" and not (m.joins == "first" and at == 0):
                    raise ValueError(f"branch {k!r} cannot share its products" + (" from this place" if m.joins else ""))
        self.scales = {k: float(v) for k, v in scales.items()} if scales is not None else None
        self.w_in = self.w_out = None
        self.spans: dict[str, tuple[int, int]] = {}       # branch -> (first column of the rows, first column of the features)
        out_norm_names = out_norm_names if out_norm_names is not None else {k: "" for k in branches}
        for k in branches:
            if k not in out_norm_names:
                raise ValueError(f"branch {k!r} needs the checkpoint name of its output norm's weight")
        self.hidden = hidden
        self.branches = dict(branches)
        self.out_norm_names = dict(out_norm_names)
        self.eps = float(eps)
        self.init_std = init_std
        self.out_weights: dict[str, torch.Tensor] = {}

    def tensor_specs(self):
        if self.scales is not None:
            return {}
        return {self.out_norm_names[k]: TensorSpec((self.hidden,), init_std=self.init_std, init_mean=1.0)
                for k in self.branches}

    def sub_parts(self):
        return list(self.branches.values())

    def cache_needs(self):
        return {f"{k}.{name}": need for k, m in self.branches.items() for name, need in m.cache_needs().items()}

    def prompt_flops(self, n_tokens: int) -> float:
        return sum(m.prompt_flops(n_tokens) for m in self.branches.values())

    def load(self, store, rt: Runtime):
        if self.scales is not None:
            return
        for k in self.branches:
            self.out_weights[k] = store.get(self.out_norm_names[k]).to(torch.float32).contiguous()

    def loaded(self, rt: Runtime):
        if self.scales is None and not self.deferred:
            return
        ins, outs, col, feat = [], [], 0, 0
        for k, m in self.branches.items():
            ins.append(m.in_weight())
            self.spans[k] = (col, feat)
            col += ins[-1].shape[0]
            if not self.deferred:
                outs.append(m.out_weight())
                feat += outs[-1].shape[1]
        if col % 8:                  # rows of the step in whole 16-byte pieces: zero rows behind the last
            ins.append(torch.zeros(8 - col % 8, self.hidden, dtype=ins[0].dtype, device=ins[0].device))
        self.w_in = torch.cat(ins, dim=0).contiguous()
        self.w_out = torch.cat(outs, dim=1).contiguous() if outs else None

    def _own(self, line, k: str) -> CacheLine:
        return CacheLine(line.index, line.write, {name[len(k) + 1:]: part for name, part in line.parts.items()
                                                  if name.startswith(k + ".")}, line.has_readers)

    def _sum(self, x, ctx: StepContext, line):
        rt, ws, T = ctx.rt, ctx.ws, ctx.n_tok
        rows = rt.linear(x, self.w_in, ws.buf("parallel.rows", (T, self.w_in.shape[0]), rt.dtype))
        z = ws.buf("parallel.z", (T, self.w_out.shape[1]), rt.dtype)
        for k, mixer in self.branches.items():
            mixer.join(rows, self.spans[k][0], ctx, self._own(line, k), z, self.spans[k][1], self.scales[k])
        return rt.linear(z, self.w_out, ws.buf("mixer.out", (T, self.hidden), rt.dtype))

    def _apart(self, x, ctx: StepContext, line) -> NormedBranches:
        rt, ws, T = ctx.rt, ctx.ws, ctx.n_tok
        rows = rt.linear(x, self.w_in, ws.buf("parallel.rows", (T, self.w_in.shape[0]), rt.dtype))
        outs = [mixer.finish(rows, self.spans[k][0], ctx, self._own(line, k), ws.buf(f"parallel.{i}", (T, self.hidden), rt.dtype))
                for i, (k, mixer) in enumerate(self.branches.items())]
        return NormedBranches(outs, [self.out_weights[k] for k in self.branches], self.eps, 1.0 / len(outs))

    def forward(self, x, ctx: StepContext, line):
        if self.scales is not None:
            return self._sum(x, ctx, line)
        if self.deferred:
            return self._apart(x, ctx, line)
        ws, ops = ctx.ws, ctx.rt.ops
        acc = ws.buf("parallel.sum", (ctx.n_tok, self.hidden), torch.float32)
        share = 1.0 / len(self.branches)
        for i, (k, mixer) in enumerate(self.branches.items()):
            r = mixer.forward(x, ctx, self._own(line, k))
            ops.rmsnorm_accumulate(r, self.out_weights[k], self.eps, share, acc, first=i == 0)
        return acc
