"""Mugedra: each mechanism against its plain statement, and the engine against the plain model.

The configurations are small and differ from each other in every size and option: grouped and ungrouped heads in both
branches; values wider and narrower than keys; turned parts of part of the head, of the whole head and none, with the ramp
and without; chunks shorter than a page, as long as one, longer, and none; capped scores and plain ones; filters of one to
five taps; key sizes of the recurrence below, at and above every border of its kernels; loops at the start, in the middle and
at the end, passed once, twice and three times, and no loop; one expert chosen and several; layers without a feed-forward;
widths that are no multiple of 4 or 8.  Weights are seeded random ones with scores spread over several units (so that attention
weights are far from uniform and the caps bite), decays from a few tokens to thousands, and write strengths from nearly 0
to nearly 1.  The bfloat16 cases read folders whose mixtures choose all their experts: a close call that rounding decides
the other way is another row of logits, not a rounding, and the recurrence carries it to every later row.  The choice itself
is compared in the float32 cases, in the router kernel's own test (which has float32 logits in both formats), and in one
bfloat16 case that is judged by its median row.

Engine cases run on the GPU (`-m gpu`, float32 and bfloat16) and, as a check of the host side alone, on the CPU over
the plain kernel statements (float32, shorter requests).
"""
from __future__ import annotations

import copy
import json
import math
import os
import subprocess
import sys

import pytest
import torch

from tests.conftest import random_tokens
from tests.helpers import assert_logits as _assert_exact, make_engine, run_in_pieces, run_requests

GPU = pytest.mark.gpu
CASES = [pytest.param("cuda", "float32", marks=GPU), pytest.param("cuda", "bfloat16", marks=GPU),
         pytest.param("refs", "float32")]
DTYPES = [torch.float32, torch.bfloat16]
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def assert_logits(got, want, dtype, what):
    """float32: every logit within 1e-4 of the largest one.  bfloat16: rows are judged by the root mean square of
    their difference against that of the logits: 19 in 20 (or all but one) within 5 %, none beyond 12 %, half of them
    within 3 %."""
    if dtype in ("float32", torch.float32):
        return _assert_exact(got, want, dtype, what)
    got, want = got.detach().double().cpu(), want.double().cpu()
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    rows = (got - want).pow(2).mean(1).sqrt() / want.pow(2).mean().sqrt()
    n = rows.numel()
    bad, worse = int((rows > 5e-2).sum()), int((rows > 12e-2).sum())
    assert bad <= max(1, n // 20) and worse == 0 and rows.median().item() < 3e-2, \
        f"{what}: {bad} of {n} rows beyond 5 %, {worse} beyond 12 %, worst {rows.max().item():.3f} at {int(rows.argmax())}, median {rows.median().item():.4f}"


def _att(heads, kv, dim, vdim, scale, chunk=0, cap=0.0, rot=0, base=10000.0, ramp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk:
        m["mask"] = {"size": chunk}
    if cap:
        m["softcap"] = cap
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if ramp:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), ramp))
    return m


def _delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def _moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def _model(vocab, width, eps, layers, loop=None):
    d = {"architecture": "Mugedra", "vocab": vocab, "width": width, "norm": {"eps": eps},
         "layers": [{"type": "parallel", "mixer": {"left": l, "right": r}, "mlp": f} for l, r, f in layers]}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# values wider than keys, short chunks, a loop over the last two of three layers
MUG_A = _model(200, 64, 1e-6, [
    (_att(4, 2, 16, 24, 0.6, chunk=10, cap=3.0, rot=8, base=1000.0, ramp=(4.0, 64, 8.0, 1.0)), _delta(4, 2, 16, 24, 4), _moe(6, 2, 24)),
    (_att(4, 1, 16, 16, 0.6, chunk=33, cap=2.0, rot=16, base=500.0), _delta(2, 2, 40, 16, 2), _moe(4, 1, 32)),
    (_att(2, 2, 32, 32, 0.4, chunk=64, cap=5.0, rot=32, base=2000.0, ramp=(16.0, 256, 4.0, 0.5)), _delta(6, 2, 24, 8, 3), None)], (1, 3, 2))

# the loop first and three times, then a layer behind it; filters of one tap; a chunk longer than a page
MUG_B = _model(333, 96, 1e-5, [
    (_att(3, 3, 16, 16, 0.7, chunk=100, cap=4.0, rot=4, base=100.0), _delta(3, 3, 36, 40, 1), _moe(4, 3, 16)),
    (_att(6, 2, 48, 48, 0.3, chunk=48, rot=48, base=300.0, ramp=(2.0, 128, 16.0, 2.0)), _delta(8, 1, 8, 48, 3), _moe(8, 2, 40))], (0, 1, 3))

# sizes a tensor-core kernel takes
MUG_C = _model(640, 128, 1e-6, [
    (_att(8, 2, 64, 64, 0.3, chunk=50, cap=6.0, rot=32, base=300000.0, ramp=(8.0, 128, 32.0, 1.0)), _delta(8, 2, 64, 64, 4), _moe(16, 4, 48)),
    (_att(4, 2, 128, 128, 0.2, chunk=130, cap=9.0), _delta(4, 4, 128, 96, 2), _moe(8, 1, 64)),
    (_att(8, 8, 32, 48, 0.4, chunk=40, cap=3.0, rot=16), _delta(4, 2, 256, 16, 4), None)], (0, 3, 1))

# sizes that are multiples of little
MUG_D = _model(301, 38, 1e-4, [
    (_att(5, 5, 10, 6, 0.8, chunk=7, cap=2.0, rot=4, base=50.0, ramp=(3.0, 32, 4.0, 1.0)), _delta(3, 1, 7, 11, 5), _moe(3, 1, 13)),
    (_att(3, 1, 6, 14, 0.9, chunk=1, cap=1.0, rot=6), _delta(2, 1, 129, 3, 4), None),
    (_att(1, 1, 2, 2, 1.0, chunk=19), _delta(4, 2, 66, 5, 3), _moe(5, 5, 6))], (1, 2, 2))

# no chunks, no cap, nothing turned, no loop
MUG_E = _model(150, 48, 1e-6, [(_att(2, 1, 16, 16, 0.7), _delta(2, 1, 200, 16, 4), _moe(3, 2, 16))])

MUG = {"A": MUG_A, "B": MUG_B, "C": MUG_C, "D": MUG_D, "E": MUG_E}


def all_experts(raw: dict) -> dict:
    """The same model with every mixture choosing all its experts."""
    raw = copy.deepcopy(raw)
    for layer in raw["layers"]:
        if layer["mlp"]:
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return raw


def write_mugedra(model_dir: str, raw: dict, seed: int, gain: float = 3.0, ff_gain: float = 8.0, router_gain: float = 8.0, zero=()) -> None:
    """A folder of seeded random weights: decays from a few tokens to thousands, write strengths spread, factors of the
    sublayers from a half to one and a half, scores of several units.  The gains suit widths of a hundred.  zero: endings of
    the names of tensors that are set to 0."""
    from janis_b200 import build_model
    from janis_b200.weights.loader import random_tensors, write_model_folder
    _, cfg, model = build_model(raw)
    tensors = random_tensors(model.tensor_specs(), seed, "cpu")
    for name, t in list(tensors.items()):
        g = torch.Generator().manual_seed(seed + len(name))
        f = None
        if name.endswith(".A_log"):
            tensors[name] = torch.linspace(-6.0, 1.0, t.numel())[torch.randperm(t.numel(), generator=g)].to(torch.bfloat16)
        elif name.endswith((".ls1", ".ls2", ".q.norm", ".k.norm")):
            tensors[name] = (0.5 + torch.rand(t.numel(), generator=g)).to(torch.bfloat16)
        elif name.endswith(".router"):
            f = router_gain
        elif name.endswith((".b", ".a")):
            f = 10.0
        elif name.endswith((".down", ".up", ".gate")):
            f = ff_gain
        elif name.endswith((".o", ".g", ".v")):
            f = gain
        if f is not None:
            tensors[name] = (t.float() * f).to(torch.bfloat16)
        if zero and name.endswith(tuple(zero)):
            tensors[name] = torch.zeros_like(tensors[name])
    write_model_folder(model_dir, cfg.to_dict(), tensors, {"seed": str(seed)})


@pytest.fixture(scope="module")
def mug_dirs(tmp_path_factory):
    out = {}
    for i, (key, raw) in enumerate(MUG.items()):
        for every in (False, True):
            d = tmp_path_factory.mktemp(f"mugedra_{key}{'_all' if every else ''}")
            write_mugedra(str(d), all_experts(raw) if every else raw, 900 + i)
            out[(key, every)] = str(d)
    return out


@pytest.fixture(scope="module")
def plain(mug_dirs):
    from tests.plain import mugedra_plain as P
    loaded, memo = {}, {}

    def logits(key, every, tokens):
        if (key, every) not in loaded:
            loaded[(key, every)] = P.load_folder(mug_dirs[(key, every)])
        k = (key, every, tuple(tokens))
        if k not in memo:
            cfg, w = loaded[(key, every)]
            memo[k] = P.forward(cfg, w, list(tokens))
        return memo[k]

    return logits


@pytest.fixture(scope="module")
def engines(mug_dirs):
    made = {}

    def get(key, dtype, on, **kw):
        every = dtype == "bfloat16"
        k = (key, dtype, on, tuple(sorted(kw.items())))
        if k not in made:
            made[k] = make_engine(mug_dirs[(key, every)], dtype, on, **kw)
        return made[k], every

    yield get
    for e in made.values():
        e.close()


def keys_for(on):
    return list(MUG) if on == "cuda" else ["A", "B", "D"]


def _requests(vocab, lens, seed):
    return [random_tokens(vocab, n, seed + i) for i, n in enumerate(lens)]


# ---------------------------------------------------------------------------
# configuration and registry
# ---------------------------------------------------------------------------

def test_configuration_reads_back_and_guards():
    from janis_b200 import ConfigError, MugedraConfig, build_model, resolve
    assert resolve(MUG_A).name == "Mugedra"
    for raw in MUG.values():
        c = MugedraConfig.from_dict(raw)
        assert MugedraConfig.from_dict(c.to_dict()) == c and c.to_dict() == {**raw, "norm": raw["norm"]}
    cfg = MugedraConfig.from_dict(MUG_A)
    assert cfg.loop.times == 2 and cfg.layers[0].mixer.left.rot_scaling.factor == 4.0 and cfg.layers[0].mixer.left.chunk == 10
    assert cfg.layers[1].mixer.left.softcap == 2.0 and cfg.layers[1].mixer.right.dim == 40 and cfg.layers[2].mlp is None
    _, _, model = build_model(MUG_A)
    specs = model.tensor_specs()
    assert specs["l0.mix.left.v"].shape == (48, 64) and specs["l0.mix.left.q.norm"].shape == (16,) and specs["l0.mix.left.g"].shape == (96, 64)
    assert specs["l0.mix.right.q"].shape == (32, 64) and specs["l0.mix.right.v.conv"].shape == (96, 4) and specs["l0.mix.right.b"].shape == (4, 64)
    assert specs["l0.mix.right.norm"].shape == (24,) and specs["l0.mix.right.out"].shape == (64,) and specs["l0.ls1"].shape == (64,)
    assert "l2.norm2" not in specs and set(model.ignorable_tensors) == {"l2.norm2", "l2.ls2"}
    assert specs["l1.mlp.router"].shape == (4, 64) and "l1.mlp.correction" not in specs and specs["l1.mlp.e3.down"].shape == (64, 32)
    assert [(c.layer, c.cache_line, c.add_embedding) for c in model.schedule] == \
        [(0, 0, False), (1, 1, False), (2, 2, False), (1, 3, True), (2, 4, False)]
    needs = model.cache_line_needs()
    assert len(needs) == 5 and set(needs[0]) == {"left.kv", "right.state", "right.conv"} and needs[3] == needs[1] != needs[2]
    _, _, model = build_model(MUG_B)
    assert [(c.layer, c.add_embedding) for c in model.schedule] == [(0, False), (0, True), (0, True), (1, False)]
    one = MUG_A["layers"][:1]
    left, right = one[0]["mixer"]["left"], one[0]["mixer"]["right"]

    def layer(l=None, r=None, f=None, **kw):
        return [{"type": "parallel", "mixer": {"left": l or left, "right": r or right}, "mlp": f, **kw}]

    for layers in (layer(type="attention"), layer({**left, "kv_heads": 3}), layer({**left, "mask": {"size": 0}}),
                   layer({**left, "rot": {"dims": 7}}), layer({**left, "rot": {"dims": 18}}), layer({**left, "softcap": -1.0}),
                   layer({**left, "rot": {"dims": 8, "scaling": {"factor": 0.0, "original": 64, "fast": 8.0, "slow": 1.0}}}),
                   layer(r={**right, "kv_heads": 3}), layer(r={**right, "conv": 0}), layer(f=_moe(4, 5, 8)),
                   layer(f={**_moe(4, 2, 8), "kind": "dense"}), [{"type": "parallel", "mixer": {"left": left}, "mlp": None}]):
        with pytest.raises(ConfigError):
            MugedraConfig.from_dict({**MUG_A, "layers": layers, "loop": None})
    for loop in ({"start": 2, "stop": 2, "times": 2}, {"start": 0, "stop": 4, "times": 2}, {"start": 0, "stop": 1, "times": 0}):
        with pytest.raises(ConfigError):
            MugedraConfig.from_dict({**MUG_A, "loop": loop})


def test_parts_refuse_what_they_cannot_do():
    from janis_b200.engine.model import LayerCall
    from janis_b200.parts import registry as parts
    names = {k: k for k in ("q", "k", "v", "o", "g", "q_norm", "k_norm")}
    pos = parts.make("position", "rotary", head_dim=8, base=10.0, rotary_dims=8)

    def attention(**kw):
        return parts.make("mixer", "talking_heads_attention", hidden=16, n_heads=2, n_kv_heads=1, key_dim=8, value_dim=8, scale=0.3,
                          position=pos, **{"names": names, "head_norm_eps": 1e-6, **kw})

    attention()
    with pytest.raises(ValueError):
        attention(head_norm_eps=None)                                    # weights without an eps
    with pytest.raises(ValueError):
        attention(names={k: k for k in ("q", "k", "v", "o", "q_norm")})  # one of the two weights
    with pytest.raises(ValueError):
        attention(names={**names, "q_bias": "qb", "k_bias": "kb", "v_bias": "vb"})
    delta_names = {k: k for k in ("q", "k", "v", "g", "b", "a", "q_conv", "k_conv", "v_conv", "A_log", "dt_bias", "norm", "o")}

    def delta(**kw):
        return parts.make("mixer", "gated_delta_rule", hidden=16, names=delta_names, norm_eps=1e-6,
                          **{"n_heads": 4, "n_key_heads": 2, "key_dim": 8, "value_dim": 8, "taps": 4, **kw})

    for bad in ({"n_key_heads": 3}, {"key_dim": 257}, {"taps": 17}, {"taps": 0}):
        with pytest.raises(ValueError):
            delta(**bad)
    with pytest.raises(ValueError):                                      # an attention's columns come first
        parts.make("mixer", "parallel", hidden=16, branches={"a": delta(), "b": attention()}, out_norm_names={"a": "x", "b": "y"}, deferred=True)
    with pytest.raises(ValueError):
        parts.make("mixer", "parallel", hidden=16, branches={"a": attention(), "b": delta()}, scales={"a": 1.0, "b": 1.0}, deferred=True)
    with pytest.raises(ValueError):
        parts.make("feed_forward", "routed_experts", hidden=8, n_experts=2, top=1, expert_ff=8, limit=0.0, scale=1.0, act="relu2",
                   weight_on="input", names={"router": "r", "expert": "e{e}.{w}"})
    from janis_b200 import build_model
    _, _, model = build_model(MUG_E)
    model.schedule[0] = LayerCall(0, 0, add_embedding=True)
    with pytest.raises(ValueError):                                      # nothing to start over
        model._check_schedule()


# ---------------------------------------------------------------------------
# the plain statements by hand
# ---------------------------------------------------------------------------

def test_plain_norms_chunks_caps_and_router_by_hand():
    from tests.plain import mugedra_plain as P
    f64 = lambda *x: torch.tensor(x, dtype=torch.float64)
    assert torch.allclose(P.layer_norm(f64(1.0, 3.0), f64(2.0, 5.0), 3.0), f64(-1.0, 2.5))         # mean 2, variance 1, root of 4
    assert torch.allclose(P.rms_norm(f64(1.0, 7.0), f64(1.0, 2.0), 0.0), f64(0.2, 2.8))
    assert torch.allclose(P.unit(f64(3.0, 4.0)), f64(0.6, 0.8), atol=1e-7)
    # chunks of two: position 2 sees itself alone, position 3 sees 2 and 3; equal scores, so the mean of their values
    z = torch.zeros(5, 1, 1, dtype=torch.float64)
    v = f64(1.0, 2.0, 4.0, 8.0, 16.0).view(5, 1, 1)
    assert torch.allclose(P.attend(z, z, v, 1.0, chunk=2).view(-1), f64(1.0, 1.5, 4.0, 6.0, 16.0))
    assert torch.allclose(P.attend(z, z, v, 1.0).view(-1), f64(1.0, 1.5, 7 / 3, 15 / 4, 31 / 5))
    # scores 0 and 100, capped at ln 3: weights 1 to 3
    q = f64(0.0, 1.0).view(2, 1, 1)
    k = f64(0.0, 100.0).view(2, 1, 1)
    assert torch.allclose(P.attend(q, k, f64(0.0, 4.0).view(2, 1, 1), 1.0, cap=math.log(3.0)).view(-1), f64(0.0, 3.0))
    idx, w = P.route(torch.log(f64(1.0, 3.0, 1.0 / 3.0)).view(1, 3), 2)
    assert idx[0].tolist() == [1, 0] and torch.allclose(w[0], f64(0.75, 0.5))                      # the scores as they are
    one = torch.ones(1, 1, dtype=torch.float64)
    w = {"gate": 2.0 * one, "up": 3.0 * one, "down": 5.0 * one}
    s = 1.0 / (1.0 + math.exp(-1.0))
    assert torch.allclose(P.expert(0.5 * one, w, ""), torch.full((1, 1), 1.0 * s * 1.5 * 5.0, dtype=torch.float64))
    full = {"router": torch.zeros(1, 1, dtype=torch.float64), **{f"e0.{k}": x for k, x in w.items()}}
    assert torch.allclose(P.moe_ff(one, full, "", {"router": {"top": 1}}), P.expert(0.5 * one, w, ""))       # the weight on the input


def test_plain_delta_rule_and_loop_by_hand():
    from tests.plain import mugedra_plain as P
    f64 = lambda *x: torch.tensor(x, dtype=torch.float64)
    k = f64([1.0, 0.0], [1.0, 0.0], [0.6, 0.8]).view(3, 1, 2)
    q = f64([1.0, 0.0], [1.0, 0.0], [0.0, 1.0]).view(3, 1, 2)
    v = f64(8.0, 2.0, 4.0).view(3, 1, 1)
    g, beta = f64(0.3, 0.5, 1.0).view(3, 1), f64(0.5, 1.0, 0.5).view(3, 1)
    # S = 4 e1 (read after the write); halved, then corrected to 2 e1; then u = (4 - 1.2) / 2 = 1.4 along (0.6, 0.8)
    assert torch.allclose(P.delta_rule(q, k, v, g, beta).view(-1), f64(4.0, 2.0, 1.12))
    assert torch.allclose(P.decay(f64(0.0), f64(math.log(2.0)), f64(0.0)), f64(0.25))              # exp(-2 ln 2)
    x = f64(1.0, 2.0, 3.0).view(3, 1)
    assert torch.allclose(P.causal_conv(x, f64([10.0, 1.0])).view(-1), f64(1.0, 12.0, 23.0))
    assert P.layer_order(4, {"start": 1, "stop": 3, "times": 2}) == [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)]
    assert P.layer_order(2, {"start": 0, "stop": 2, "times": 1}) == P.layer_order(2, None) == [(0, False), (1, False)]


def test_planted_mistakes_in_the_oracle_show(mug_dirs):
    """A loop that does not add the embedding again, chunks one position longer, caps left out, weights on the experts' outputs,
    weights that add up to 1, a state read before its write: each moves the logits far beyond any tolerance here."""
    from tests.plain import mugedra_plain as P
    cfg, w = P.load_folder(mug_dirs[("A", False)])
    toks = random_tokens(cfg["vocab"], 60, 3)
    right = P.forward(cfg, w, toks)

    def on_output(y, w_, pre, mlp):
        idx, wts = P.route(y @ w_[pre + "router"].T, mlp["router"]["top"])
        return torch.stack([sum(a * P.expert(y[t:t + 1], w_, f"{pre}e{e}.")[0] for e, a in zip(idx[t].tolist(), wts[t])) for t in range(y.shape[0])])

    def stale(q, k, v, g, beta):
        S, out = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=torch.float64), torch.zeros_like(v)
        for t in range(q.shape[0]):
            S = g[t][:, None, None] * S
            out[t] = torch.einsum("hdv,hd->hv", S, q[t])
            S = S + k[t][:, :, None] * (beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t])))[:, None, :]
        return out

    real = {n: getattr(P, n) for n in ("layer_order", "attend", "route", "moe_ff", "delta_rule")}
    planted = {
        "no embedding": ("layer_order", lambda n, loop: [(i, False) for i, _ in real["layer_order"](n, loop)]),
        "longer chunks": ("attend", lambda q, k, v, scale, cap=0.0, chunk=0: real["attend"](q, k, v, scale, cap, chunk + 1)),
        "no cap": ("attend", lambda q, k, v, scale, cap=0.0, chunk=0: real["attend"](q, k, v, scale, 0.0, chunk)),
        "on the output": ("moe_ff", on_output),
        "renormalized": ("route", lambda z, top: (lambda i, x: (i, x / x.sum(-1, keepdim=True)))(*real["route"](z, top))),
        "stale state": ("delta_rule", stale)}
    for what, (name, wrong) in planted.items():
        setattr(P, name, wrong)
        try:
            moved = (P.forward(cfg, w, toks) - right).abs().max().item()
        finally:
            setattr(P, name, real[name])
        assert moved > 0.05 * right.abs().max().item(), (what, moved)


# ---------------------------------------------------------------------------
# kernels against their statements
# ---------------------------------------------------------------------------

def _close(got, want, dtype, what, f32=2e-5, bf16=2e-2):
    tol = f32 if dtype == torch.float32 else bf16
    err = (got.cpu().double() - want.double()).abs().max().item()
    assert math.isfinite(err) and err <= tol * max(1.0, want.double().abs().max().item()), (what, err)


def _tables(lens, starts, slots):
    tok_pos, tok_seq, first = [], [], []
    for s, (n, st) in enumerate(zip(lens, starts)):
        first.append(len(tok_pos))
        tok_pos += list(range(st, st + n))
        tok_seq += [s] * n
    i32 = lambda x: torch.tensor(x, dtype=torch.int32)
    return (i32(tok_pos), i32(tok_seq), i32(slots), i32(first), i32(starts), i32([a + b for a, b in zip(starts, lens)]))


def _cuda(*xs):
    return tuple(x.cuda() if x is not None else None for x in xs)


@GPU
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,rot,amp", [(4, 2, 16, 24, 8, 1.2), (5, 5, 10, 6, 4, 1.0), (3, 1, 6, 14, 0, 1.0), (8, 8, 96, 64, 48, 1.3),
                                              (2, 1, 64, 128, 64, 1.4), (6, 3, 48, 16, 48, 1.0), (16, 2, 256, 256, 128, 1.1), (1, 1, 2, 2, 2, 2.0)])
def test_norm_turn_store_kernel_against_its_statement(dtype, H, G, d, dv, rot, amp):
    """Sequences that start, that go on across a page's border, one token, and a padding sequence; heads of very different
    lengths (the norm takes them out), one nearly zero; columns behind q, k and v stay."""
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    g = torch.Generator().manual_seed(5)
    lens, starts, slots = [7, 1, 70, 3, 2], [0, 63, 60, 5, 0], [2, 0, 4, 1, -1]
    tok_pos, tok_seq, seq_slot, *_ = _tables(lens, starts, slots)
    T = sum(lens)
    per = max(-(-(a + n) // ops.PAGE) for a, n in zip(starts, lens))
    table = torch.randperm(5 * per, generator=g).view(5, per).to(torch.int32)
    cols = H * d + G * (d + dv)
    for tail in (3, (-cols) % 8 + 8):                         # rows that rule 16-byte loads out, and rows that allow them
        rows = torch.randn(T, cols + tail, generator=g)
        rows[:, :(H + G) * d] *= torch.logspace(-1, 1, H + G).repeat_interleave(d)
        rows[4, :d] = 1e-4
        rows = rows.to(dtype)
        wq, wk = torch.rand(d, generator=g) + 0.5, torch.rand(d, generator=g) - 1.5
        inv = torch.rand(rot // 2, generator=g) * 2
        kp, vp = torch.zeros(5 * per, G, ops.PAGE, d, dtype=dtype), torch.zeros(5 * per, G, ops.PAGE, dv, dtype=dtype)
        want_rows, wkp, wvp = rows.clone(), kp.clone(), vp.clone()
        extras = dict(amplitude=amp, norm_eps=1e-3)
        R.qkv_rotate_store(want_rows, tok_pos, tok_seq, seq_slot, inv, rot, None, H, G, d, dv, wkp, wvp, table, q_norm=wq, k_norm=wk, **extras)
        got_rows, gk, gv = _cuda(rows, kp, vp)
        ops.qkv_rotate_store(got_rows, *_cuda(tok_pos, tok_seq, seq_slot, inv), rot, None, H, G, d, dv, gk, gv, table.cuda(),
                             q_norm=wq.cuda(), k_norm=wk.cuda(), **extras)
        for got, want, what in ((got_rows, want_rows, "rows"), (gk, wkp, "keys"), (gv, wvp, "values")):
            _close(got, want, dtype, (what, tail), f32=5e-5)
        assert torch.equal(got_rows[:, cols:].cpu(), rows[:, cols:])


def _hot_keys(kp, q, spots, d):
    """Key 0 of the given (page, place) pairs and the first head of every query get a large score together."""
    hot = torch.zeros(d, dtype=torch.float32)
    hot[0] = 4.0
    q[:, :d] = (q[:, :d].float() * 0.2 + hot).to(q.dtype)
    for page, place in spots:
        kp[page, 0, place] = hot.to(kp.dtype)


@GPU
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,chunk", [(4, 2, 16, 24, 10), (8, 8, 96, 64, 64), (5, 5, 10, 6, 7), (16, 2, 16, 64, 100), (6, 1, 48, 128, 1), (8, 4, 128, 64, 65)])
def test_capped_attention_in_chunks_against_its_statement(dtype, H, G, d, dv, chunk):
    """On the tensor cores (rows together; a row a CTA; a row's keys over 3 CTAs), in the plain kernel and in the kernels that
    take single rows.  Keys that stand out lie just outside and just inside the chunks of the queries around their edges."""
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    lens = [1, 70, 129, 300]
    g = torch.Generator().manual_seed(3)
    per = -(-300 // ops.PAGE)
    table = torch.randperm(6 * per, generator=g).view(6, per).to(torch.int32)
    slots = torch.tensor([4, 1, 0, 5], dtype=torch.int32)
    kp, vp = torch.randn(6 * per, G, ops.PAGE, d, generator=g).to(dtype), torch.randn(6 * per, G, ops.PAGE, dv, generator=g).to(dtype)
    pos, seq = [], []
    for s, n in enumerate(lens):
        edges = {0, n - 1, n // 2, 63, 64, chunk - 1, chunk, chunk + 1, 2 * chunk - 1, 2 * chunk}
        for p in sorted(p for p in edges if p < n):
            pos.append(p)
            seq.append(s)
    T = len(pos)
    q = torch.randn(T, H * d + (-H * d) % 8, generator=g).to(dtype)
    _hot_keys(kp, q, [(int(table[int(slots[s]), j // ops.PAGE]), j % ops.PAGE) for s in range(4) for j in (0, chunk - 1, chunk, 2 * chunk - 1) if j < lens[s]], d)
    tok_pos, tok_seq = torch.tensor(pos, dtype=torch.int32), torch.tensor(seq, dtype=torch.int32)
    scale, cap = 0.5, 2.5
    want, open_, uncapped = (torch.zeros(T, H * dv, dtype=dtype) for _ in range(3))
    R.talk_attention(q, tok_pos, tok_seq, slots, kp, vp, table, None, None, want, H, G, d, dv, scale, chunk, cap=cap)
    R.talk_attention(q, tok_pos, tok_seq, slots, kp, vp, table, None, None, open_, H, G, d, dv, scale, chunk + 1, cap=cap)
    R.talk_attention(q, tok_pos, tok_seq, slots, kp, vp, table, None, None, uncapped, H, G, d, dv, scale, chunk)
    assert (want.float() - open_.float()).abs().max().item() > 0.2
    assert chunk == 1 or (want.float() - uncapped.float()).abs().max().item() > 0.2
    dq, dpos, dseq, dslot, dk, dv_, dtab = _cuda(q, tok_pos, tok_seq, slots, kp, vp, table)
    for which, one_row, chunks in ((1, False, 1), (1, True, 1), (1, True, 3), (0, False, 1)):
        ops.talk_attention_set_kernel(which)
        try:
            got = torch.full((T, H * dv), float("nan"), dtype=dtype, device="cuda")
            n = ops.talk_attention_scratch_floats(T, chunks, H, dv)
            scratch = torch.full((n,), float("nan"), device="cuda") if n else None
            ops.talk_attention(dq, dpos, dseq, dslot, dk, dv_, dtab, None, None, got, H, G, d, dv, scale, chunk, one_row=one_row,
                               max_keys=min(chunk, 300), n_chunks=chunks, scratch=scratch, cap=cap)
        finally:
            ops.talk_attention_set_kernel(1)
        _close(got, want, dtype, (which, one_row, chunks))
    n = ops.talk_attention_rows_floats(dtype, T, H, G, d, dv, chunk)
    vec = 4 if dtype == torch.float32 else 8
    assert (n > 0) == (d % vec == 0 and dv % vec == 0)
    if n:
        got = torch.full((T, H * dv), float("nan"), dtype=dtype, device="cuda")
        ops.talk_attention_rows(dq, dpos, dseq, dslot, dk, dv_, dtab, None, got, H, G, d, dv, scale,
                                torch.full((n,), float("nan"), device="cuda"), chunk, window=-chunk, cap=cap)
        _close(got, want, dtype, "rows")


@GPU
@pytest.mark.parametrize("H,G,d,chunk,cap", [(4, 2, 16, 10, 2.0), (8, 8, 64, 50, 3.0), (8, 4, 128, 64, 0.0), (6, 2, 48, 130, 5.0), (4, 2, 256, 33, 2.0),
                                             (16, 1, 128, 1, 1.0), (2, 2, 64, 129, 4.0), (2, 1, 64, 5000, 4.0)])
def test_kernels_of_whole_heads_in_chunks_with_a_cap(H, G, d, chunk, cap):
    """Prompt steps (every form of the kernels; sequences that start and sequences that go on from stored keys) and decode
    steps (a row's keys in one piece and in several) around the edges of chunks, with keys that stand out there."""
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    dtype = torch.bfloat16
    g = torch.Generator().manual_seed(13)
    width = ((H + 2 * G) * d + 9 + 7) // 8 * 8
    scale = 2.0 * d ** -0.5

    def case(lens, starts):
        tok_pos, tok_seq, slots, first, start, end = _tables(lens, starts, [len(lens) - s for s in range(len(lens))])
        per = max(-(-(a + n) // ops.PAGE) for a, n in zip(starts, lens))
        n_slots = len(lens) + 1
        table = torch.randperm(n_slots * per, generator=g).view(n_slots, per).to(torch.int32)
        kp = torch.randn(n_slots * per, G, ops.PAGE, d, generator=g).to(dtype)
        vp = torch.randn(n_slots * per, G, ops.PAGE, d, generator=g).to(dtype)
        rows = torch.randn(sum(lens), width, generator=g).to(dtype)
        _hot_keys(kp, rows, [(int(table[int(slots[s]), j // ops.PAGE]), j % ops.PAGE) for s in range(len(lens))
                             for j in (0, chunk - 1, chunk) if j < starts[s]], d)
        for t, p in enumerate(tok_pos.tolist()):
            if p in (0, chunk - 1, chunk):
                rows[t, H * d:(H + 1) * d] = torch.tensor([4.0] + [0.0] * (d - 1)).to(dtype)
        R.qkv_rotate_store(rows, tok_pos, tok_seq, slots, torch.zeros(0), 0, None, H, G, d, d, kp, vp, table)
        return tok_pos, tok_seq, slots, first, start, end, table, kp, vp, rows

    def statement(c, size):
        tok_pos, tok_seq, slots, first, start, end, table, kp, vp, rows = c
        want = torch.zeros(rows.shape[0], H * d, dtype=dtype)
        R.talk_attention(rows, tok_pos, tok_seq, slots, kp, vp, table, None, None, want, H, G, d, d, scale, size, cap=cap)
        return want

    for lens, starts in (([1, 65, 290], [0] * 3), ([70, 2, 150], [70, 129, 31])):
        c = case(lens, starts)
        tok_pos, tok_seq, slots, first, start, end, table, kp, vp, rows = c
        before = dict(seq_start=start.cuda(), seq_slot=slots.cuda(), kpool=kp.cuda(), vpool=vp.cuda(), page_table=table.cuda()) if any(starts) else {}
        T = rows.shape[0]
        n = ops.attn_prefill_scratch_floats(T, len(lens), H, d, dtype)
        want = statement(c, chunk)
        if chunk < 200:
            assert (want.float() - statement(c, chunk + 1).float()).abs().max().item() > 0.2
        for which in (0, 1, 2, 3):
            for piece in (0, 1):
                ops.attn_set_prefill_kernel(d, which)
                ops.attn_set_prefill_piece(d, piece)
                try:
                    got = torch.full((T, H * d), float("nan"), dtype=dtype, device="cuda")
                    ops.attn_prefill_rows(rows.cuda(), first.cuda(), end.cuda(), got, H, G, d, scale, -chunk, cap=cap,
                                          scratch=torch.full((max(n, 1),), float("nan"), device="cuda") if n else None,
                                          host_lens=tuple(lens) if which != 2 else None, **before)
                finally:
                    ops.attn_set_prefill_kernel(d, 1)
                    ops.attn_set_prefill_piece(d, 0)
                _close(got, want, dtype, ("prompt", lens, which, piece))
        assert ops.attn_tc05_timeouts(d) == 0
    at = [0, chunk - 1, chunk, 2 * chunk - 1, 2 * chunk, 299]
    c = case([1] * 6, [min(p, 299) for p in at])
    tok_pos, tok_seq, slots, first, start, end, table, kp, vp, rows = c
    want = statement(c, chunk)
    for piece in (64, 128, 320):
        pieces = min(-(-320 // piece), -(-chunk // piece) + 1)
        scratch = torch.full((ops.attn_decode_scratch_floats(6, H, d, pieces),), float("nan"), device="cuda")
        got = torch.full((6, H * d), float("nan"), dtype=dtype, device="cuda")
        ops.attn_decode_rows(*_cuda(rows, kp, vp, table, slots, end), scratch, got, H, G, d, scale, -chunk, piece, pieces, cap=cap)
        _close(got, want, dtype, ("decode", piece))
    assert ops.attn_wait_timeouts(d) == 0


def _delta_case(H, G, d, dv, T, dtype, seed, pad=5):
    """Convolved rows (q, k, v from column 3 on), projected rows (gate, b, a from column 2 on) and the heads' constants."""
    g = torch.Generator().manual_seed(seed)
    C = 2 * G * d + H * dv
    x = torch.randn(T, 3 + C + pad, generator=g)
    x[:, 3:3 + 2 * G * d] *= torch.rand(T, 1, generator=g) * 3 + 0.1             # (the unit norm takes the length out)
    z = 2.0 * torch.randn(T, 2 + H * dv + 2 * H + pad, generator=g)
    return dict(x=x.to(dtype), z=z.to(dtype), offs=(3, 3 + G * d, 3 + 2 * G * d), g_off=2, b_off=2 + H * dv, a_off=2 + H * dv + H,
                decay=-torch.exp(torch.linspace(-6.0, 1.0, H)), dt_bias=torch.randn(H, generator=g), w=torch.rand(dv, generator=g) + 0.5), g


DELTA_SIZES = [(4, 2, 16, 24), (3, 1, 7, 11), (8, 2, 64, 64), (4, 4, 128, 96), (2, 1, 129, 3), (4, 2, 256, 16), (6, 6, 66, 5), (2, 2, 36, 20), (16, 8, 128, 128)]


@GPU
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv", DELTA_SIZES)
def test_delta_rule_kernels_against_their_statements(dtype, H, G, d, dv):
    """Prompts that end at, just before and just after the kernel's blocks of four tokens and its tiles, sequences that go on from
    a stored state, one token, a padding sequence; states of untouched slots stay; one and two columns a group of lanes, many
    short sequences.  Then steps of single rows with the head's norm and gate, and a prompt's own norm and gate beside them."""
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    runs = [([8, 1, 7, 9, 2, 16, 17, 3, 35], [0, 9, 4, 0, 0, 0, 77, 0, 2])]
    if d <= 16:
        runs.append(([2, 5] * 80, [0, 3] * 80))
    for lens, starts in runs:
        T, ns = sum(lens), len(lens)
        slots = [s if s != 7 else -1 for s in range(ns)]
        tok_pos, tok_seq, *tabs = _tables(lens, starts, slots)
        c, g = _delta_case(H, G, d, dv, T, dtype, 21)
        state = torch.randn(ns + 2, H, dv, d, generator=g)
        for st, slot in zip(starts, slots):
            if st == 0 and slot >= 0:
                state[slot] = 0.0
        want, ws = torch.zeros(T, H * dv), state.clone()
        args = (c["a_off"], c["b_off"])
        R.delta_scan(c["x"], *c["offs"], c["z"], *args, c["decay"], c["dt_bias"], d ** -0.5, tok_pos, tok_seq, *tabs, ws, want, ns, H, G, d, dv)
        for form in (0, 1, 2):
            got, gs = torch.full((T, H * dv), float("nan"), device="cuda"), state.cuda()
            coef = torch.full((T, H, ops.DELTA_COEF), float("nan"), device="cuda")
            ops.delta_scan(c["x"].cuda(), *c["offs"], c["z"].cuda(), *args, *_cuda(c["decay"], c["dt_bias"]), d ** -0.5, *_cuda(tok_pos, tok_seq, *tabs),
                           gs, got, ns, H, G, d, dv, coef, form=form)
            _close(got, want, torch.float32, ("scan", form, ns))           # (float from the convolved rows on, whatever they are stored in)
            _close(gs, ws, torch.float32, ("states", form, ns))
            assert torch.equal(gs[ns:].cpu(), state[ns:])
    for T in (1, 8, 13):
        c, g = _delta_case(H, G, d, dv, T, dtype, 23)
        tok_seq = torch.arange(T, dtype=torch.int32)
        slots = torch.randperm(T + 2, generator=g)[:T].to(torch.int32)
        if T > 1:
            slots[T // 2] = -1
        state = torch.randn(T + 2, H, dv, d, generator=g)
        want, ws, got, gs = torch.zeros(T, H * dv, dtype=dtype), state.clone(), torch.full((T, H * dv), float("nan"), dtype=dtype, device="cuda"), state.cuda()
        args = (c["a_off"], c["b_off"], c["g_off"])
        R.delta_step(c["x"], *c["offs"], c["z"], *args, c["decay"], c["dt_bias"], d ** -0.5, c["w"], 1e-5, tok_seq, slots, ws, want, H, G, d, dv)
        ops.delta_step(c["x"].cuda(), *c["offs"], c["z"].cuda(), *args, *_cuda(c["decay"], c["dt_bias"]), d ** -0.5, c["w"].cuda(), 1e-5,
                       *_cuda(tok_seq, slots), gs, got, H, G, d, dv)
        _close(got, want, dtype, ("step", T), bf16=1e-2)
        _close(gs, ws, torch.float32, ("states", T))


@GPU
@pytest.mark.parametrize("cuts", [(0, 4096), (0, 1, 3, 700, 701, 3001, 4096)])
def test_a_state_that_remembers_thousands_of_tokens_keeps_its_last_bits(cuts):
    """Decays just below 1 over 4,096 tokens, small write strengths: an error of one sign in every step (g rounded to a float)
    would add up to 1e-4 of the state; and the same tokens in pieces of uneven sizes leave the same state."""
    from janis_b200.kernels import ops
    H, d, dv, T = 8, 16, 4, 4096
    g = torch.Generator().manual_seed(4)
    x = torch.cat([torch.randn(T, H * d, generator=g), torch.randn(T, H * d, generator=g) + 0.3, torch.rand(T, H * dv, generator=g) + 0.5], 1)
    decay = -torch.logspace(-6.0, -3.0, H)
    z = torch.cat([torch.zeros(T, H), torch.full((T, H), -6.0)], 1)
    gate = torch.exp(decay.double() * math.log(2.0))
    k = x[:, H * d:2 * H * d].double().view(T, H, d)
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    v, beta = x[:, 2 * H * d:].double().view(T, H, dv), 1.0 / (1.0 + math.exp(6.0))
    S = torch.zeros(H, dv, d, dtype=torch.float64)
    for t in range(T):
        S = S * gate[:, None, None]
        S = S + (beta * (v[t] - torch.einsum("hvd,hd->hv", S, k[t])))[:, :, None] * k[t][:, None, :]
    i32 = lambda *v_: torch.tensor(v_, dtype=torch.int32, device="cuda")
    state = torch.zeros(1, H, dv, d, device="cuda")
    for lo, hi in zip(cuts, cuts[1:]):
        n = hi - lo
        ops.delta_scan(x[lo:hi].cuda().contiguous(), 0, H * d, 2 * H * d, z[lo:hi].cuda().contiguous(), 0, H, decay.cuda(), torch.zeros(H, device="cuda"), 1.0,
                       torch.arange(lo, hi, dtype=torch.int32, device="cuda"), torch.zeros(n, dtype=torch.int32, device="cuda"), i32(0), i32(0), i32(lo), i32(hi),
                       state, torch.zeros(n, H * dv, device="cuda"), 1, H, H, d, dv, torch.zeros(n, H, ops.DELTA_COEF, device="cuda"))
    err = (state[0].cpu().double() - S).abs().amax((1, 2)) / S.abs().amax((1, 2))
    assert err.max().item() < 5e-6, err.tolist()


@GPU
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [38, 64, 96, 1000, 1024, 1540, 2304, 3584, 4608, 6144, 6148, 2305])
def test_sum_into_the_stream_with_the_norm_behind_it_against_its_statement(dtype, W):
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    g = torch.Generator().manual_seed(W)
    T = 7
    h = 3.0 * torch.randn(T, W, generator=g) + 5.0                       # a mean far from zero
    r = [(torch.randn(T, W, generator=g) * s).to(dtype) for s in (0.3, 4.0)]
    more, vec = torch.randn(T, W, generator=g), lambda: torch.rand(W, generator=g) + 0.5
    bw, scale, w_next = [vec(), vec()], vec(), vec()
    for kw in (dict(r=r[0], w=True), dict(r=r[0], scale=scale, w=True, centred=True), dict(r=r[0], scale=scale, more=more, w=True, centred=True),
               dict(r=r, branch_weights=bw, eps=1e-3, share=0.5, scale=scale, w=True, centred=True),
               dict(r=r, branch_weights=bw, eps=1e-3, share=0.5, scale=scale, more=more, w=True, centred=True),
               dict(r=r[:1], branch_weights=bw[:1], eps=1e-3, share=1.0, w=True), dict(r=r, branch_weights=bw, eps=1e-3, share=0.5, scale=scale), dict(r=more),
               dict(w=True, centred=True), dict(rows=torch.tensor([6, 0, 0, 3, 1], dtype=torch.int32), w=True, centred=True)):
        kw = dict(kw)
        has = kw.pop("w", False)
        R_ = len(kw["rows"]) if "rows" in kw else T
        want_h, got_h = h.clone(), h.cuda()
        want = torch.zeros(R_, W, dtype=dtype) if has else None
        got = torch.full((R_, W), float("nan"), dtype=dtype, device="cuda") if has else None
        more_kw = dict(w_next=w_next, eps_next=1e-3) if has else {}
        R.stream_norm(want_h, out=want, **kw, **more_kw)
        dev = lambda v: [x.cuda() for x in v] if isinstance(v, list) else (v.cuda() if torch.is_tensor(v) else v)
        ops.stream_norm(got_h, out=got, **{k: dev(v) for k, v in kw.items()}, **{k: dev(v) for k, v in more_kw.items()})
        _close(got_h, want_h, torch.float32, (sorted(kw), "stream"), f32=2e-6)
        if has:
            _close(got, want, dtype, (sorted(kw), "norm"), f32=1e-5, bf16=1e-2)
        if "r" not in kw:
            assert torch.equal(got_h.cpu(), h)


@GPU
@pytest.mark.parametrize("E,top", [(3, 1), (16, 4), (5, 5), (1, 1), (64, 6), (200, 3)])
def test_router_of_plain_scores_and_experts_weighted_on_their_input_against_their_statements(E, top):
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    from tests.plain import mugedra_plain as P
    g = torch.Generator().manual_seed(6)
    T = 53
    z = 3.0 * torch.randn(T, E, generator=g)
    want = torch.zeros(T, E)
    R.moe_route(z, None, E, 1, 1, top, 1.0, False, want, raw=True)
    got = torch.full((T, E), float("nan"), device="cuda")
    ops.moe_route(z.cuda(), None, E, 1, 1, top, 1.0, False, got, raw=True)
    assert torch.equal(got.cpu() != 0, want != 0)
    _close(got, want, torch.float32, "weights")
    idx, w = P.route(z.double(), top)
    _close(got, torch.zeros(T, E, dtype=torch.float64).scatter_(1, idx, w), torch.float32, "weights of the plain model")
    inf = float("inf")
    for dtype in DTYPES:
        for ff in (16, 13):
            gu = (3.0 * torch.randn(T, 2 * E * ff, generator=g)).to(dtype)
            out, other = torch.zeros(T, E * ff, dtype=dtype), torch.zeros(T, E * ff, dtype=dtype)
            R.moe_expert_act(gu, want, E, ff, inf, 0, inf, 1.0, out, up_add=0.0, weight_in=True)
            R.moe_expert_act(gu, want, E, ff, inf, 0, inf, 1.0, other, up_add=0.0)
            assert (out.float() - other.float()).abs().max().item() > 0.02
            a = torch.full((T, E * ff), float("nan"), dtype=dtype, device="cuda")
            ops.moe_expert_act(gu.cuda(), got, E, ff, inf, 0, inf, 1.0, a, up_add=0.0, weight_in=True)
            _close(a, out, dtype, ("experts", ff))


# ---------------------------------------------------------------------------
# the engine against the plain model
# ---------------------------------------------------------------------------

@pytest.mark.parametrize("on,dtype", CASES)
def test_whole_prompts_and_first_tokens(engines, plain, on, dtype):
    for key in keys_for(on):
        eng, every = engines(key, dtype, on, max_tokens=2048)
        lens = [1, 2, 3, 70, 150] if on == "cuda" else [1, 2, 40]
        reqs = _requests(MUG[key]["vocab"], lens, 11)
        got = run_requests(eng, reqs, lens)
        for r, g_ in zip(reqs, got):
            assert_logits(g_, plain(key, every, r), dtype, f"{key} whole {len(r)}")


@pytest.mark.parametrize("on,dtype", CASES)
def test_prompts_of_unequal_lengths_then_decoded_together(engines, plain, on, dtype):
    """Batches one after another, so that slots, pages and states are used again; a request of one token beside long ones;
    decoding carries the recurrence and the filter over their stored states and the attention across pages and chunks."""
    for key in keys_for(on):
        eng, every = engines(key, dtype, on, max_tokens=2048)
        if on == "cuda":
            lens, prompts = [260, 1, 140, 67, 200, 30], [120, 1, 60, 64, 63, 5]
        else:
            lens, prompts = [40, 1, 30, 12], [20, 1, 6, 9]
        reqs = _requests(MUG[key]["vocab"], lens, 23)
        got = run_requests(eng, reqs, prompts, max_live=3 if on == "cuda" else 2)
        for r, g_ in zip(reqs, got):
            assert_logits(g_, plain(key, every, r), dtype, f"{key} batch {len(r)}")


@pytest.mark.parametrize("on,dtype", CASES)
def test_a_request_alone_and_in_company_and_token_by_token(engines, plain, on, dtype):
    for key in keys_for(on)[:4]:
        eng, every = engines(key, dtype, on, max_tokens=2048)
        n = 90 if on == "cuda" else 25
        reqs = _requests(MUG[key]["vocab"], [n, 17, n // 2], 31)
        alone = run_requests(eng, reqs[:1], [n // 3])[0]
        together = run_requests(eng, reqs, [n // 3, 9, 4])[0]
        one_by_one = run_requests(eng, reqs[:1], [1])[0]
        want = plain(key, every, reqs[0])
        for g_, what in ((alone, "alone"), (together, "in company"), (one_by_one, "token by token")):
            assert_logits(g_, want, dtype, f"{key} {what}")
        if dtype == "float32" and on == "cuda":
            assert (alone - together).abs().max().item() <= 1e-4 * want.abs().max().item()


@pytest.mark.parametrize("on,dtype", CASES)
@pytest.mark.parametrize("chunk", [2, 3, 16, 64, 65])
def test_prompts_in_pieces(engines, plain, on, dtype, chunk):
    if on == "refs" and chunk > 16:
        pytest.skip("long pieces run on the GPU")
    for key in keys_for(on)[:4]:
        eng, every = engines(key, dtype, on, max_tokens=2048)
        lens = [150, 66, 7] if on == "cuda" else [21, 9]
        reqs = _requests(MUG[key]["vocab"], lens, 41)
        got = run_in_pieces(eng, reqs, chunk)
        for r, g_ in zip(reqs, got):
            assert_logits(g_, plain(key, every, r), dtype, f"{key} pieces of {chunk}, {len(r)} tokens")


@GPU
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_recorded_steps(engines, plain, dtype):
    for key in ("A", "C"):
        eng, every = engines(key, dtype, "cuda", max_tokens=2048)
        reqs = _requests(MUG[key]["vocab"], [330, 300], 51)
        got = run_requests(eng, reqs, [10, 3])
        for r, g_ in zip(reqs, got):
            assert_logits(g_, plain(key, every, r), dtype, f"{key} long decoding")


@GPU
def test_chosen_experts_in_the_serving_type(mug_dirs, plain):
    """Mixtures that choose, in bfloat16: close calls move single rows and, through the recurrence, some that follow; half of
    all rows stay within the rounding."""
    for key in ("A", "B", "C", "D"):
        eng = make_engine(mug_dirs[(key, False)], "bfloat16", "cuda", max_tokens=2048)
        try:
            reqs = _requests(MUG[key]["vocab"], [90] * 6, 55)
            want = [plain(key, False, r) for r in reqs]
            rows = torch.cat([(g_.double() - w).pow(2).mean(1).sqrt() / w.pow(2).mean().sqrt()
                              for g_, w in zip(run_requests(eng, reqs, [60] * 6), want)])
            assert rows.median().item() < 3e-2 and (rows < 5e-2).double().mean().item() > 0.6, (key, rows.median().item())
        finally:
            eng.close()


@GPU
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_step_writes_what_it_reads(engines, plain, dtype):
    """Prompt steps of one padded shape (launched, recorded, replayed) and decode steps with every scratch buffer full of NaN
    before each; padding rows stand in both."""
    from janis_b200 import StepEntry
    for key in ("A", "B", "D"):
        eng, every = engines(key, dtype, "cuda", max_tokens=2048)
        V = MUG[key]["vocab"]
        for b, lens in enumerate([(30, 45, 9), (33, 40, 10), (20, 50, 5)]):
            reqs = _requests(V, [n + 3 for n in lens], 81 + b)
            slots = [eng.alloc_slot() for _ in reqs]
            eng.stepper.ws.fill(float("nan"))
            rows = [eng.step([StepEntry(s, r[:n], [n - 1]) for s, r, n in zip(slots, reqs, lens)])]
            for t in range(3):
                eng.stepper.ws.fill(float("nan"))
                rows.append(eng.step([StepEntry(s, [r[n + t]], [0]) for s, r, n in zip(slots, reqs, lens)]))
            for i, (r, n) in enumerate(zip(reqs, lens)):
                assert_logits(torch.stack([x[i] for x in rows]), plain(key, every, r)[n - 1:n + 3], dtype, f"{key} batch {b} request {i}")
            for s in slots:
                eng.free_slot(s)


@pytest.mark.parametrize("on,dtype", CASES)
def test_keys_just_inside_and_just_outside_a_chunk(tmp_path_factory, on, dtype):
    """One layer whose recurrence is silenced: a token changed at a chunk's last position moves no logits of the next chunk
    (not by a bit) and one changed at a chunk's first position moves those of its last; in a prompt, in pieces, decoded."""
    chunk = 20
    d = str(tmp_path_factory.mktemp("mugedra_edge"))
    write_mugedra(d, _model(120, 64, 1e-6, [(_att(2, 1, 16, 16, 0.5, chunk=chunk, cap=4.0, rot=8), _delta(2, 1, 16, 16, 4), None)]), 78, zero=(".right.o",))
    eng = make_engine(d, dtype, on, max_tokens=1024)
    try:
        base = random_tokens(120, 3 * chunk, 6)
        ways = {"whole": lambda r: run_requests(eng, [r], [len(r)])[0], "decoded": lambda r: run_requests(eng, [r], [5])[0],
                "pieces": lambda r: run_in_pieces(eng, [r], 7)[0]}
        for what, run in ways.items():
            a = run(base)
            for at in (chunk - 1, chunk, 2 * chunk - 1):
                b = run(base[:at] + [(base[at] + 1) % 120] + base[at + 1:])
                moved = (a - b).abs().amax(1)
                end = (at // chunk + 1) * chunk
                assert moved[:at].max().item() == 0.0 and moved[end:].max().item() == 0.0, (what, at)
                assert moved[at:end].min().item() > 1e-3, (what, at, moved[at:end].tolist())
    finally:
        eng.close()


@GPU
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_first_token_far_back_reaches_the_end_through_the_recurrence_alone(tmp_path_factory, dtype):
    """One layer whose attention sees chunks of 30: the first of 260 tokens reaches the end through the state, and not without."""
    for silenced in (".left.o", ".right.o"):
        d = str(tmp_path_factory.mktemp("mugedra_far"))
        write_mugedra(d, _model(120, 64, 1e-6, [(_att(2, 1, 16, 16, 0.5, chunk=30), _delta(6, 3, 32, 16, 4), None)]), 78, zero=(silenced, ".right.b"))
        eng = make_engine(d, dtype, "cuda", max_tokens=1024)
        try:
            base = random_tokens(120, 260, 6)
            other = [(base[0] + 1) % 120] + base[1:]
            for n in (260, 200):
                a, b = (run_requests(eng, [r], [n])[0][-1] for r in (base, other))
                moved = (a - b).abs().max().item()
                assert moved == 0.0 if silenced == ".right.o" else moved > (1e-5 if dtype == "float32" else 0.0), (silenced, n, moved)
        finally:
            eng.close()


def test_branches_left_to_the_block_are_the_branches_own(mug_dirs):
    """The parallel mixer's one input product, and the sum that the block's kernel makes of its branches, against the branches run
    one by one, normed and averaged (the plain kernel statements, float32), in a prompt step."""
    from janis_b200.parts.base import StepContext
    from janis_b200.parts.norm import NormedBranches
    outs = []
    for apart in (False, True):
        eng = make_engine(mug_dirs[("B", False)], "float32", "refs", max_tokens=512)
        mixer = eng.model.blocks[1].mixer
        T, W = 11, MUG_B["width"]
        x = torch.randn(T, W, generator=torch.Generator().manual_seed(2))
        slot = eng.alloc_slot()
        eng.cache.reserve(slot, T)
        eng.cache.sync()
        tok_pos, tok_seq, slots, first, start, end = _tables([T], [0], [slot])
        ctx = StepContext(rt=eng.rt, ws=eng.stepper.ws, mode="prefill", n_tok=T, n_seq=1, tokens=tok_pos, tok_pos=tok_pos, tok_seq=tok_seq,
                          seq_slot=slots, seq_start=start, seq_end=end, seq_first_row=first, len_bound=T)
        line = eng.cache.line(3, True)
        h = torch.zeros(T, W)
        if apart:
            cut = [mixer.spans[k][0] for k in mixer.branches] + [mixer.w_in.shape[0]]
            mixer.branches["left"].w_qkv, mixer.branches["right"].w_in = (mixer.w_in[a:b].contiguous() for a, b in zip(cut, cut[1:]))
            mixer.deferred = False
            h += mixer.forward(x, ctx, line)
        else:
            r = mixer.forward(x, ctx, line)
            assert isinstance(r, NormedBranches)
            eng.rt.ops.stream_norm(h, r.parts, branch_weights=r.weights, eps=r.eps, share=r.share)
        outs.append(h)
    assert (outs[0] - outs[1]).abs().max().item() < 1e-5 * outs[1].abs().max().item()


@pytest.mark.parametrize("on,dtype", CASES)
def test_greedy_generation_through_the_engine(engines, plain, on, dtype):
    for key in ("A", "B"):
        eng, every = engines(key, dtype, on, max_tokens=2048)
        prompts = _requests(MUG[key]["vocab"], [33, 5, 70] if on == "cuda" else [9, 4], 61)
        n_new = 8 if on == "cuda" else 4
        replies = eng.generate(prompts, temp=0.0, max_tokens=n_new, stop=())
        assert all(len(r) == n_new for r in replies)
        for p, r in zip(prompts, replies):
            seq = list(p)
            for tok in r:
                logits = plain(key, every, seq)[-1]
                assert logits[tok] >= logits.max() - (1e-4 if dtype == "float32" else 4e-2) * logits.abs().max(), (key, len(seq))
                seq.append(tok)


@GPU
def test_trace_replay_and_command_line_as_a_user_runs_them(mug_dirs, plain, tmp_path):
    key, every = "A", False
    reqs = _requests(MUG[key]["vocab"], [40, 9], 71)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": reqs[0][:30], "want": [0, 29]}, {"id": "b", "tokens": reqs[1][:5], "want": [4]}], "end": []}]
    for i in range(10):
        ents = [{"id": "a", "tokens": [reqs[0][30 + i]], "want": [0]}]
        if 5 + i < 9:
            ents.append({"id": "b", "tokens": [reqs[1][5 + i]], "want": [0]})
        steps.append({"step": i + 1, "entries": ents, "end": ["b"] if 5 + i == 8 else (["a"] if i == 9 else [])})
    out = tmp_path / "out"
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", mug_dirs[(key, every)], "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(11)]
    import numpy as np
    V = MUG[key]["vocab"]
    wa, wb = plain(key, every, reqs[0]), plain(key, every, reqs[1])
    first = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(-1, V).copy())
    assert_logits(first, torch.stack([wa[0], wa[29], wb[4]]), "float32", "trace step 0")
    for i in range(10):
        got = torch.from_numpy(np.fromfile(out / f"{i + 1}.f32", dtype="<f4").reshape(-1, V).copy())
        want = [wa[30 + i]] + ([wb[5 + i]] if 5 + i < 9 else [])
        assert_logits(got, torch.stack(want), "float32", f"trace step {i + 1}")
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "janis"), "generate", "--model", mug_dirs[(key, every)], "--dtype", "float32",
                        "--ids", ",".join(map(str, reqs[1])), "--max-tokens", "4", "--temp", "0", "--stop", ""],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    seq = list(reqs[1])
    for _ in range(4):
        seq.append(int(plain(key, every, seq)[-1].argmax()))
    assert ",".join(map(str, seq[len(reqs[1]):])) in p.stdout.replace(" ", ""), p.stdout


def test_the_comparison_model_of_the_benchmark_builds_at_every_size():
    from janis_b200 import MugedraConfig, build_model
    from janis_b200.benchmark import mugedra_like, load_config
    for name in ("gemma2-2b", "gemma2-9b", "gemma2-27b"):
        gemma = load_config(name)
        raw = mugedra_like(gemma, 4)
        cfg = MugedraConfig.from_dict(raw)
        assert [l.type for l in cfg.layers] == ["parallel"] * 4
        _, _, model = build_model(raw)
        assert model.hidden == gemma["hidden_size"] and model.vocab == gemma["vocab_size"]
        assert all(n.shape for n in model.tensor_specs().values() if n.shape != ())


# two layers, passed twice, at sizes that reach the launch shapes, vector loads and library products the small models do not
MUG_WIDE = _model(2048, 1024, 1e-6, [
    (_att(8, 2, 128, 128, 0.3, chunk=200, cap=20.0, rot=64, base=100000.0, ramp=(8.0, 256, 32.0, 1.0)), _delta(16, 8, 128, 128, 4), _moe(8, 2, 512)),
    (_att(8, 4, 128, 64, 0.3, chunk=300, cap=10.0, rot=128, base=100000.0), _delta(8, 2, 64, 128, 4), _moe(8, 2, 512))], (0, 2, 2))


@GPU
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_looped_layers_at_the_sizes_of_a_larger_model(tmp_path_factory, dtype):
    from tests.plain import mugedra_plain as P
    d = str(tmp_path_factory.mktemp("mugedra_wide"))
    write_mugedra(d, all_experts(MUG_WIDE) if dtype == "bfloat16" else MUG_WIDE, 91, gain=1.0, ff_gain=2.0, router_gain=2.0)
    cfg, w = P.load_folder(d)
    eng = make_engine(d, dtype, "cuda", max_tokens=4096)
    try:
        reqs = _requests(MUG_WIDE["vocab"], [560, 300, 40], 95)
        got = run_requests(eng, reqs, [520, 270, 3])
        for r, g_ in zip(reqs, got):
            assert_logits(g_, P.forward(cfg, w, r), dtype, f"wide {len(r)}")
    finally:
        eng.close()
