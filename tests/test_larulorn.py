"""Larulorn: each mechanism against its plain statement, and the engine against the plain model.

The configurations are small and differ from each other in every size and option: every order of the two mixers; layers
whose values are mixed and layers whose are not, one mixing layer alone and several apart; grouped and ungrouped heads;
values wider and narrower than keys; turned parts of four features, of part of the head, of the whole head and none, with
the ramp and without; one block of gates and several, filters of one to five taps; constants of the two branches that
differ; routers with groups of one, two and four, groups of one expert and no groups, one expert chosen and several, with and
without a shared expert; layers without a feed-forward; widths that are no multiple of 8.  Weights are seeded random ones
with the projections of queries and keys scaled up, so that the attention weights are far from uniform, sinks spread around
the scores, and decays spread, so that some channels of the recurrence forget within a few tokens and others remember
hundreds.  The bfloat16 cases read folders whose mixtures choose all their experts: a close call that rounding decides the
other way is another row of logits, not a rounding, and the recurrence carries it to every later row.  The choice itself is
compared in the float32 cases, in the router kernel's own test (which has float32 logits in both formats), and in one
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


def _att(heads, kv, dim, vdim, scale, rot=0, base=10000.0, ramp=None, v_mix=False):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if ramp:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), ramp))
    if v_mix:
        m["v_mix"] = True
    return m


def _par(left, width, blocks, conv, left_scale, right_scale):
    return {"left": left, "right": {"width": width, "blocks": blocks, "conv": conv}, "left_scale": left_scale,
            "right_scale": right_scale}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(experts, top, ff, groups=None, shared=0):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r, "shared": {"ff": shared} if shared else None}


def _model(vocab, width, eps, logit, layers):
    return {"architecture": "Larulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit,
            "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in layers]}


# values wider than keys, mixed in two layers with a parallel layer between them; a layer whose values are its own; groups
LAR_A = _model(200, 64, 1e-6, 1.25, [
    ("attention", _att(4, 2, 16, 24, 0.25, rot=8, base=1000.0, ramp=(4.0, 64, 8.0, 1.0), v_mix=True), _dense(40, 1.0)),
    ("parallel", _par(_att(4, 1, 16, 16, 0.3, rot=16, base=500.0), 48, 3, 4, 0.7, 0.4), _moe(6, 2, 24, (3, 2), shared=40)),
    ("attention", _att(6, 2, 16, 24, 0.25, rot=16, base=1000.0, ramp=(16.0, 256, 4.0, 0.5), v_mix=True), None),
    ("attention", _att(2, 2, 32, 16, 0.2, rot=32), _moe(5, 3, 16))])

# a parallel layer first: nothing turned, one block of gates, a filter of one tap; a layer that says it mixes alone; one
# expert chosen, groups of one expert, one group kept
LAR_B = _model(333, 96, 1e-5, 0.5, [
    ("parallel", _par(_att(3, 3, 16, 32, 0.25), 32, 1, 1, 1.0, 1.5), _moe(4, 1, 32, (2, 1))),
    ("attention", _att(6, 6, 16, 8, 0.3, rot=4, base=100.0, v_mix=True), _dense(72, 0.5)),
    ("parallel", _par(_att(6, 2, 32, 16, 0.2, rot=8, base=300000.0), 80, 5, 3, -0.5, 2.0), None),
    ("attention", _att(4, 1, 48, 24, 0.15, rot=48, base=300.0, ramp=(2.0, 128, 16.0, 2.0)), _moe(4, 2, 16, (4, 3), shared=8))])

# sizes a tensor-core kernel takes; three layers that mix, no constant on the logits
LAR_C = _model(640, 128, 1e-6, 1.0, [
    ("attention", _att(8, 2, 64, 64, 0.12, rot=32, base=300000.0, ramp=(8.0, 128, 32.0, 1.0), v_mix=True), _moe(16, 4, 48, (4, 2), shared=80)),
    ("attention", _att(16, 2, 16, 64, 0.25, rot=16, v_mix=True), _dense(160, 2.0)),
    ("parallel", _par(_att(8, 8, 32, 48, 0.2, rot=16), 256, 2, 2, 0.3, 0.9), _moe(8, 2, 64, (8, 3))),
    ("attention", _att(4, 2, 96, 64, 0.1, rot=64, base=2000.0, ramp=(32.0, 512, 32.0, 1.0), v_mix=True), _dense(96, 7.0))])

# sizes that are multiples of little
LAR_D = _model(301, 36, 1e-4, 3.0, [
    ("attention", _att(5, 5, 10, 6, 0.3, rot=4, base=50.0, ramp=(3.0, 32, 4.0, 1.0), v_mix=True), _dense(21, 0.8)),
    ("parallel", _par(_att(3, 1, 6, 14, 0.4, rot=6), 21, 3, 5, 0.9, 0.6), _moe(3, 1, 13, shared=5)),
    ("attention", _att(10, 5, 12, 6, 0.3, v_mix=True), _moe(9, 3, 7, (3, 1))),
    ("parallel", _par(_att(1, 1, 2, 2, 0.7, rot=2), 10, 2, 4, 0.25, 1.0), None)])

# each mixer alone, without a feed-forward
LAR_E = _model(150, 48, 1e-6, 1.0, [("parallel", _par(_att(2, 1, 16, 16, 0.3, rot=8), 64, 4, 4, 0.5, 0.5), None)])
LAR_F = _model(97, 40, 1e-5, 2.0, [("attention", _att(2, 1, 16, 8, 0.3, rot=16, ramp=(8.0, 64, 8.0, 1.0), v_mix=True), None)])

LAR = {"A": LAR_A, "B": LAR_B, "C": LAR_C, "D": LAR_D, "E": LAR_E, "F": LAR_F}


def all_experts(raw: dict) -> dict:
    """The same model with every mixture choosing all its experts."""
    raw = copy.deepcopy(raw)
    for layer in raw["layers"]:
        if layer["mlp"] and layer["mlp"]["kind"] == "moe":
            r = layer["mlp"]["router"]
            r["top"] = r["experts"]
            if "groups" in r:
                r["groups"]["keep"] = r["groups"]["count"]
    return raw


def write_larulorn(model_dir: str, raw: dict, seed: int, gain: float = 3.0, qk_gain: float = 6.0, router_gain: float = 30.0,
                   sink_gain: float = 2.0) -> None:
    """A folder of seeded random weights: query and key projections and biases scaled up (peaked attention weights), sinks
    spread, decays from a few tokens to thousands, gates and up matrices that reach the limits.  The gains suit widths of a
    hundred."""
    from janis_b200 import build_model
    from janis_b200.weights.loader import random_tensors, write_model_folder
    _, cfg, model = build_model(raw)
    tensors = random_tensors(model.tensor_specs(), seed, "cpu")
    for name, t in list(tensors.items()):
        g = torch.Generator().manual_seed(seed + len(name))
        f = None
        if name.endswith((".q", ".k", ".q.b", ".k.b")):
            f = qk_gain
        elif name.endswith(".sink"):
            f = sink_gain
        elif name.endswith(".v.b"):
            f = 10.0
        elif name.endswith(".lam"):
            tensors[name] = torch.linspace(-9.0, 1.0, t.numel())[torch.randperm(t.numel(), generator=g)].to(torch.bfloat16)
        elif name.endswith(".router"):
            f = router_gain
        elif name.endswith((".o", ".down", ".up", ".gate", ".g", ".v", ".mix.right.x", ".mix.right.y")):
            f = gain
        if f is not None:
            tensors[name] = (t.float() * f).to(torch.bfloat16)
    write_model_folder(model_dir, cfg.to_dict(), tensors, {"seed": str(seed)})


@pytest.fixture(scope="module")
def lar_dirs(tmp_path_factory):
    out = {}
    for i, (key, raw) in enumerate(LAR.items()):
        for every in (False, True):
            d = tmp_path_factory.mktemp(f"larulorn_{key}{'_all' if every else ''}")
            write_larulorn(str(d), all_experts(raw) if every else raw, 800 + i)
            out[(key, every)] = str(d)
    return out


@pytest.fixture(scope="module")
def plain(lar_dirs):
    from tests.plain import larulorn_plain as P
    loaded, memo = {}, {}

    def logits(key, every, tokens):
        if (key, every) not in loaded:
            loaded[(key, every)] = P.load_folder(lar_dirs[(key, every)])
        k = (key, every, tuple(tokens))
        if k not in memo:
            cfg, w = loaded[(key, every)]
            memo[k] = P.forward(cfg, w, list(tokens))
        return memo[k]

    return logits


@pytest.fixture(scope="module")
def engines(lar_dirs):
    made = {}

    def get(key, dtype, on, **kw):
        every = dtype == "bfloat16"
        k = (key, dtype, on, tuple(sorted(kw.items())))
        if k not in made:
            made[k] = make_engine(lar_dirs[(key, every)], dtype, on, **kw)
        return made[k], every

    yield get
    for e in made.values():
        e.close()


def keys_for(on):
    return list(LAR) if on == "cuda" else ["A", "B", "D", "E", "F"]


def _requests(vocab, lens, seed):
    return [random_tokens(vocab, n, seed + i) for i, n in enumerate(lens)]


# ---------------------------------------------------------------------------
# configuration and registry
# ---------------------------------------------------------------------------

def test_configuration_reads_back_and_guards():
    from janis_b200 import ConfigError, LarulornConfig, build_model, resolve
    cfg = LarulornConfig.from_dict(LAR_A)
    assert LarulornConfig.from_dict(cfg.to_dict()) == cfg
    assert resolve(LAR_A).name == "Larulorn"
    assert cfg.logit_scale == 1.25 and cfg.layers[0].mixer.rot_scaling.factor == 4.0 and cfg.layers[0].mixer.v_mix
    assert cfg.layers[1].mixer.left_scale == 0.7 and cfg.layers[1].mixer.right.blocks == 3 and cfg.layers[2].mlp is None
    assert cfg.layers[1].mlp.group_count == 3 and cfg.layers[1].mlp.group_keep == 2 and cfg.layers[3].mlp.group_count == 1
    for raw in LAR.values():
        c = LarulornConfig.from_dict(raw)
        assert LarulornConfig.from_dict(c.to_dict()) == c
    _, _, model = build_model(LAR_A)
    specs = model.tensor_specs()
    assert specs["l0.mix.v"].shape == (48, 64) and specs["l0.mix.q.b"].shape == (64,) and specs["l0.mix.sink"].shape == (4,)
    assert "l0.mix.vmix" not in specs and "l0.mix.vmix" in model.ignorable_tensors      # the first mixing layer's number is unused
    assert specs["l2.mix.vmix"].shape == () and "l2.mix.vmix" not in model.ignorable_tensors and "l3.mix.vmix" in model.ignorable_tensors
    assert specs["l1.mix.left.g"].shape == (64, 64) and "l1.mix.left.sink" not in specs and "l1.mix.left.q.b" not in specs
    assert specs["l1.mix.right.ra"].shape == (3, 16, 16) and specs["l1.mix.right.conv"].shape == (48, 4) and specs["l1.mix.right.lam"].shape == (48,)
    assert specs["l0.norm1b"].shape == (64,) and "l2.norm2b" not in specs and "l2.norm2b" in model.ignorable_tensors
    assert specs["l1.mlp.router"].shape == (6, 64) and "l1.mlp.e0.gate" not in specs and "l1.mlp.shared.sg" not in specs
    assert "l1.mlp.correction" not in specs and "l3.mlp.shared.up" not in specs and specs["l1.mlp.shared.down"].shape == (64, 40)
    needs = model.cache_line_needs()
    assert set(needs[0]) == {"kv"} and needs[0]["kv"].n_kv_heads == 2 and needs[0]["kv"].value_dim == 24
    assert set(needs[1]) == {"left.kv", "right.state", "right.conv"} and needs[1]["right.state"].shape == (48,)
    bad_layers = [
        [{"type": "conv", "mixer": {}, "mlp": None}],
        [{"type": "attention", "mixer": _att(4, 3, 32, 32, 0.2), "mlp": None}],
        [{"type": "attention", "mixer": _att(4, 2, 32, 32, 0.2, rot=34), "mlp": None}],
        [{"type": "attention", "mixer": _att(4, 2, 32, 32, 0.2, rot=7), "mlp": None}],
        [{"type": "attention", "mixer": _att(4, 2, 32, 32, 0.2, rot=8, ramp=(0.0, 64, 8.0, 1.0)), "mlp": None}],
        [{"type": "attention", "mixer": _att(4, 2, 32, 32, 0.2, v_mix=True), "mlp": None},
         {"type": "attention", "mixer": _att(4, 4, 32, 32, 0.2, v_mix=True), "mlp": None}],
        [{"type": "parallel", "mixer": _par(_att(2, 1, 16, 16, 0.2), 50, 4, 4, 1.0, 1.0), "mlp": None}],
        [{"type": "parallel", "mixer": _par(_att(2, 1, 16, 16, 0.2, v_mix=True), 48, 4, 4, 1.0, 1.0), "mlp": None}],
        [{"type": "attention", "mixer": _att(2, 1, 16, 16, 0.2), "mlp": _dense(32, 0.0)}],
        [{"type": "attention", "mixer": _att(2, 1, 16, 16, 0.2), "mlp": _moe(6, 2, 8, (4, 2))}],
        [{"type": "attention", "mixer": _att(2, 1, 16, 16, 0.2), "mlp": _moe(6, 3, 8, (3, 1))}],
        [{"type": "attention", "mixer": _att(2, 1, 16, 16, 0.2), "mlp": {**_dense(8, 1.0), "kind": "sparse"}}]]
    for layers in bad_layers:
        with pytest.raises(ConfigError):
            LarulornConfig.from_dict({**LAR_A, "layers": layers})


def test_parts_refuse_what_they_cannot_do():
    from janis_b200.parts import registry as parts
    pos = parts.make("position", "rotary", head_dim=8, base=10.0, rotary_dims=8)
    names = {k: k for k in ("q", "k", "v", "o", "g")}

    def attention(**kw):
        return parts.make("mixer", "talking_heads_attention", hidden=16, n_heads=2, n_kv_heads=1, key_dim=8, value_dim=8, scale=0.3,
                          position=pos, **{"names": names, **kw})

    with pytest.raises(ValueError):
        attention(names={**names, "q_bias": "q.b"})                      # biases on one projection alone
    with pytest.raises(ValueError):
        attention(value_mix="mix")                                       # no number to mix with
    rec = parts.make("mixer", "gated_recurrence", hidden=16, width=8, blocks=2, taps=4, names={
        k: k for k in ("y", "y_bias", "x", "x_bias", "conv", "conv_bias", "ra", "ra_bias", "ri", "ri_bias", "lam", "o")})
    with pytest.raises(ValueError):                                      # an attention's columns come first
        parts.make("mixer", "parallel", hidden=16, branches={"a": rec, "b": attention()}, scales={"a": 1.0, "b": 1.0})
    with pytest.raises(ValueError):
        parts.make("mixer", "parallel", hidden=16, branches={"a": attention(), "b": rec}, scales={"a": 1.0})
    with pytest.raises(ValueError):
        parts.make("feed_forward", "gated_mlp", hidden=8, intermediate=8, names={k: k for k in ("gate", "up", "down")}, act="clamped_swish")


# ---------------------------------------------------------------------------
# the plain statements by hand
# ---------------------------------------------------------------------------

def test_plain_positions_sink_values_and_router_by_hand():
    from tests.plain import larulorn_plain as P
    f, amp = P.frequencies({"base": 100.0, "dims": 4})
    assert amp == 1.0 and torch.allclose(f, torch.tensor([1.0, 0.1], dtype=torch.float64))
    # the ramp: 4 dims, base e^2: a pair of t turns stands at ln(original / (2 pi t)); fast = original / (2 pi): 0, slow: 1
    base, orig = math.exp(2.0), 2.0 * math.pi * 50.0
    f, amp = P.frequencies({"base": base, "dims": 4, "scaling": {"factor": 10.0, "original": orig, "fast": 50.0, "slow": 50.0 / math.e}})
    assert abs(amp - (0.1 * math.log(10.0) + 1.0)) < 1e-15
    assert torch.allclose(f, torch.tensor([1.0, math.exp(-1.0) / 10.0], dtype=torch.float64))      # kept, stretched
    x = torch.tensor([[[1.0, 0.0, 0.0, 1.0, 5.0]]], dtype=torch.float64).repeat(2, 1, 1)
    y = P.turn(x, torch.arange(2), torch.tensor([1.0, 2.0], dtype=torch.float64), 3.0)
    c1, s1, c2, s2 = math.cos(1), math.sin(1), math.cos(2), math.sin(2)
    assert torch.allclose(y[1, 0], torch.tensor([3 * c1, -3 * s2, 3 * s1, 3 * c2, 5.0], dtype=torch.float64))     # pairs (0, 2) and (1, 3)
    assert torch.allclose(y[0, 0], torch.tensor([3.0, 0.0, 0.0, 3.0, 5.0], dtype=torch.float64))
    # one key of score 0, sink ln 3: the key keeps a quarter
    one = torch.zeros(1, 1, 2, dtype=torch.float64)
    v = torch.tensor([[[8.0]]], dtype=torch.float64)
    assert torch.allclose(P.attend(one, one, v, 1.0, torch.tensor([math.log(3.0)], dtype=torch.float64)), torch.tensor([[[2.0]]], dtype=torch.float64))
    assert torch.allclose(P.attend(one, one, v, 1.0), v)
    assert torch.allclose(P.mix_values(torch.tensor(2.0), torch.tensor(10.0), 0.25), torch.tensor(4.0))
    # the router: groups of two; the second group holds the best entry and the worst, the third the two middle ones
    z = torch.log(torch.tensor([[0.05, 0.1, 0.4, 0.01, 0.24, 0.2]], dtype=torch.float64))
    idx, w = P.route(z, 2, {"count": 3, "keep": 1})
    assert sorted(idx[0].tolist()) == [2, 3] and abs(float(w.sum()) - 1.0) < 1e-12
    idx, w = P.route(z, 2, {"count": 3, "keep": 2})
    assert sorted(idx[0].tolist()) == [2, 4] and abs(dict(zip(idx[0].tolist(), w[0].tolist()))[2] - 0.4 / 0.64) < 1e-12
    assert sorted(P.route(z, 3)[0][0].tolist()) == [2, 4, 5]


def test_plain_recurrence_filter_and_feed_forwards_by_hand():
    from tests.plain import larulorn_plain as P
    # gates at 1/2, softplus(lam) = ln 2 / 4: log a = -8 / 2 * ln 2 / 4 = -ln 2, a = 1/2
    lam = torch.log(torch.expm1(torch.tensor([math.log(2.0) / 4.0], dtype=torch.float64)))
    half = torch.full((3, 1), 0.5, dtype=torch.float64)
    u = torch.tensor([[4.0], [0.0], [8.0]], dtype=torch.float64)
    S = P.linear_recurrence(u, half, half, lam)
    k = 0.5 * math.sqrt(0.75)
    assert torch.allclose(S[:, 0], torch.tensor([4 * k, 2 * k, 9 * k], dtype=torch.float64))        # the first token like any other
    x = torch.tensor([[1.0], [2.0], [3.0]], dtype=torch.float64)
    out = P.causal_conv(x, torch.tensor([[10.0, 1.0]], dtype=torch.float64), torch.tensor([0.5], dtype=torch.float64))
    assert torch.allclose(out[:, 0], torch.tensor([1.5, 12.5, 23.5], dtype=torch.float64))
    mats = torch.zeros(2, 1, 1, dtype=torch.float64)
    mats[1] = 1.0
    z = P.block_gate(torch.tensor([[5.0, 2.0]], dtype=torch.float64), mats, torch.tensor([[0.0], [1.0]], dtype=torch.float64))
    assert torch.allclose(z, torch.tensor([[0.5, 1 / (1 + math.exp(-3.0))]], dtype=torch.float64))
    one = torch.ones(1, 1, dtype=torch.float64)
    w = {"gate": 9.0 * one, "up": -9.0 * one, "down": one}
    g = 1.5 / (1 + math.exp(-1.702 * 1.5))
    assert torch.allclose(P.clamped_gate(one, w, "", 1.5), torch.tensor([[g * (-1.5 + 1.0)]], dtype=torch.float64))
    assert torch.allclose(P.clamped_gate(-one, w, "", 100.0), torch.tensor([[-9.0 / (1 + math.exp(1.702 * 9.0)) * 10.0]], dtype=torch.float64))
    assert torch.allclose(P.expert(one, {"up": 3.0 * one, "down": 2.0 * one}, ""), 18.0 * one)
    assert torch.allclose(P.expert(-one, {"up": 3.0 * one, "down": 2.0 * one}, ""), 0.0 * one)


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
@pytest.mark.parametrize("H,G,d,dv,rot,amp,bias,mix", [
    (4, 2, 16, 24, 8, 1.2, True, 1), (4, 2, 16, 24, 8, 1.2, True, 2), (5, 5, 10, 6, 4, 1.0, True, 2), (3, 1, 6, 14, 0, 1.0, True, 0),
    (8, 8, 96, 64, 48, 1.3, True, 2), (2, 1, 64, 128, 64, 1.4, False, 1), (6, 3, 48, 16, 48, 1.0, False, 2), (1, 1, 2, 2, 2, 2.0, True, 1)])
def test_bias_turn_mix_store_kernel_against_its_statement(dtype, H, G, d, dv, rot, amp, bias, mix):
    """Sequences that start, that go on across a page's border, one token, and a padding sequence; the rows, the values left
    for later layers and both pools are compared."""
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    g = torch.Generator().manual_seed(5)
    lens, starts, slots = [7, 1, 70, 3, 2], [0, 63, 60, 5, 0], [2, 0, 4, 1, -1]
    tok_pos, tok_seq, seq_slot, *_ = _tables(lens, starts, slots)
    T = sum(lens)
    per = max(-(-(a + n) // ops.PAGE) for a, n in zip(starts, lens))
    table = torch.randperm(5 * per, generator=g).view(5, per).to(torch.int32)
    cols = H * d + G * (d + dv)
    rows = torch.randn(T, cols + 3, generator=g).to(dtype)
    b = torch.randn(cols, generator=g) if bias else None
    first = torch.randn(T, G * dv, generator=g).to(dtype)
    inv = torch.rand(rot // 2, generator=g) * 2
    kp, vp = torch.zeros(5 * per, G, ops.PAGE, d, dtype=dtype), torch.zeros(5 * per, G, ops.PAGE, dv, dtype=dtype)
    want_rows, want_first, wk, wv = rows.clone(), first.clone(), kp.clone(), vp.clone()
    extras = dict(amplitude=amp, mix=mix, share=0.3)
    R.qkv_rotate_store(want_rows, tok_pos, tok_seq, seq_slot, inv, rot, None, H, G, d, dv, wk, wv, table, bias=b, v_first=want_first, **extras)
    got_rows, got_first, gk, gv = _cuda(rows, first, kp, vp)
    ops.qkv_rotate_store(got_rows, *_cuda(tok_pos, tok_seq, seq_slot, inv), rot, None, H, G, d, dv, gk, gv, table.cuda(),
                         bias=b.cuda() if bias else None, v_first=got_first, **extras)
    for got, want, what in ((got_rows, want_rows, "rows"), (got_first, want_first, "first"), (gk, wk, "keys"), (gv, wv, "values")):
        _close(got, want, dtype, what, f32=5e-5)
    if mix == 1:
        assert torch.equal(got_first.view(T, -1), got_rows[:, H * d + G * d:cols])
    elif mix == 0:
        assert torch.equal(got_first.cpu(), first)


@GPU
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 16, 24), (8, 8, 96, 64), (5, 5, 10, 6), (16, 2, 16, 64), (6, 1, 48, 128), (8, 4, 128, 128)])
def test_attention_with_learnt_sinks_against_its_statement(dtype, H, G, d, dv):
    """On the tensor cores (rows together; a row a CTA; a row's keys over 3 and 7 CTAs), in the plain kernel and in the kernels
    that take single rows.  Under head 0 the sequence's very first key, and one at a page's border, get a large score; head
    1's sink is larger than its scores, head 2's tiny: leaving the sinks out would show."""
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    lens = [1, 70, 129, 300]
    g = torch.Generator().manual_seed(3)
    per = [-(-n // ops.PAGE) for n in lens]
    n_pages = sum(per) + 3
    order = torch.randperm(n_pages, generator=g).tolist()
    table, slots, at = torch.zeros(6, max(per), dtype=torch.int32), torch.tensor([4, 1, 0, 5], dtype=torch.int32), 0
    for s in range(4):
        for j in range(per[s]):
            table[int(slots[s]), j] = order[at]
            at += 1
    kp = torch.randn(n_pages, G, ops.PAGE, d, generator=g).to(dtype)
    vp = torch.randn(n_pages, G, ops.PAGE, dv, generator=g).to(dtype)
    pos, seq = [], []
    for s, n in enumerate(lens):
        for p in sorted({0, n - 1, n // 2, min(n - 1, 63), min(n - 1, 64), min(n - 1, 128)}):
            pos.append(p)
            seq.append(s)
    T = len(pos)
    q = torch.randn(T, H * d + (-H * d) % 8, generator=g).to(dtype)
    hot = torch.zeros(d)
    hot[0] = 5.0
    q[:, :d] = (q[:, :d].float() * 0.2 + hot).to(dtype)
    for s in range(4):
        for j in (0, 64):
            if j < lens[s]:
                kp[int(table[int(slots[s]), j // ops.PAGE]), 0, j % ops.PAGE] = hot.to(dtype)
    sinks = torch.randn(H, generator=g)
    sinks[1 % H] = 6.0
    if H > 2:
        sinks[2] = -30.0
    tok_pos, tok_seq = torch.tensor(pos, dtype=torch.int32), torch.tensor(seq, dtype=torch.int32)
    scale = 0.3
    want, without = torch.zeros(T, H * dv, dtype=dtype), torch.zeros(T, H * dv, dtype=dtype)
    R.talk_attention(q, tok_pos, tok_seq, slots, kp, vp, table, None, None, want, H, G, d, dv, scale, 0, True, sink_values=sinks)
    R.talk_attention(q, tok_pos, tok_seq, slots, kp, vp, table, None, None, without, H, G, d, dv, scale, 0, False)
    assert (want.float() - without.float()).abs().max().item() > 0.05
    dq, dpos, dseq, dslot, dk, dv_, dtab, dsink = _cuda(q, tok_pos, tok_seq, slots, kp, vp, table, sinks)
    for which, one_row, chunks in ((1, False, 1), (1, True, 1), (1, True, 3), (1, True, 7), (0, False, 1)):
        ops.talk_attention_set_kernel(which)
        try:
            got = torch.full((T, H * dv), float("nan"), dtype=dtype, device="cuda")
            n = ops.talk_attention_scratch_floats(T, chunks, H, dv)
            scratch = torch.full((n,), float("nan"), device="cuda") if n else None
            ops.talk_attention(dq, dpos, dseq, dslot, dk, dv_, dtab, None, None, got, H, G, d, dv, scale, 0, True, one_row=one_row,
                               max_keys=300, n_chunks=chunks, scratch=scratch, sink_values=dsink)
        finally:
            ops.talk_attention_set_kernel(1)
        _close(got, want, dtype, (which, one_row, chunks))
    for bound in (300, 5000):
        n = ops.talk_attention_rows_floats(dtype, T, H, G, d, dv, bound)
        vec = 4 if dtype == torch.float32 else 8
        assert (n > 0) == (d % vec == 0 and dv % vec == 0)
        if n:
            got = torch.full((T, H * dv), float("nan"), dtype=dtype, device="cuda")
            ops.talk_attention_rows(dq, dpos, dseq, dslot, dk, dv_, dtab, None, got, H, G, d, dv, scale,
                                    torch.full((n,), float("nan"), device="cuda"), bound, sink=True, sink_values=dsink)
            _close(got, want, dtype, ("rows", bound))


@GPU
@pytest.mark.parametrize("H,G,d,window", [(4, 2, 16, 0), (8, 8, 64, 50), (8, 4, 128, 0), (6, 2, 48, 130), (4, 2, 256, 0), (16, 1, 192, 0)])
def test_kernels_of_whole_heads_over_longer_rows_with_learnt_sinks(H, G, d, window):
    """Prompt steps (every form of the kernels; sequences that start and sequences that go on from stored keys) and decode
    steps (a row's keys in one chunk and in several), with columns behind q, k and v, with and without sinks."""
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    dtype = torch.bfloat16
    g = torch.Generator().manual_seed(13)
    width = ((H + 2 * G) * d + 9 + 7) // 8 * 8
    scale = 2.0 * d ** -0.5
    sinks = torch.randn(H, generator=g)
    sinks[0], sinks[1] = 6.0, -30.0

    def case(lens, starts):
        tok_pos, tok_seq, slots, first, start, end = _tables(lens, starts, [len(lens) - s for s in range(len(lens))])
        per = max(-(-(a + n) // ops.PAGE) for a, n in zip(starts, lens))
        n_slots = len(lens) + 1
        table = torch.randperm(n_slots * per, generator=g).view(n_slots, per).to(torch.int32)
        kp = torch.randn(n_slots * per, G, ops.PAGE, d, generator=g).to(dtype)
        vp = torch.randn(n_slots * per, G, ops.PAGE, d, generator=g).to(dtype)
        rows = torch.randn(sum(lens), width, generator=g).to(dtype)
        R.qkv_rotate_store(rows, tok_pos, tok_seq, slots, torch.zeros(0), 0, None, H, G, d, d, kp, vp, table)
        return tok_pos, tok_seq, slots, first, start, end, table, kp, vp, rows

    def statement(c, z):
        tok_pos, tok_seq, slots, first, start, end, table, kp, vp, rows = c
        want = torch.zeros(rows.shape[0], H * d, dtype=dtype)
        R.talk_attention(rows, tok_pos, tok_seq, slots, kp, vp, table, None, None, want, H, G, d, d, scale, 0, z is not None,
                         window=window, sink_values=z)
        return want

    for lens, starts in (([1, 65, 140], [0] * 3), ([70, 2], [70, 129])):
        c = case(lens, starts)
        tok_pos, tok_seq, slots, first, start, end, table, kp, vp, rows = c
        before = dict(seq_start=start.cuda(), seq_slot=slots.cuda(), kpool=kp.cuda(), vpool=vp.cuda(), page_table=table.cuda()) if any(starts) else {}
        T = rows.shape[0]
        n = ops.attn_prefill_scratch_floats(T, len(lens), H, d, dtype)
        for z in (sinks, None):
            want = statement(c, z)
            for which in (0, 1, 2, 3):
                for piece in (0, 1):
                    ops.attn_set_prefill_kernel(d, which)
                    ops.attn_set_prefill_piece(d, piece)
                    try:
                        got = torch.full((T, H * d), float("nan"), dtype=dtype, device="cuda")
                        ops.attn_prefill_rows(rows.cuda(), first.cuda(), end.cuda(), got, H, G, d, scale, window,
                                              sinks=z.cuda() if z is not None else None,
                                              scratch=torch.full((max(n, 1),), float("nan"), device="cuda") if n else None,
                                              host_lens=tuple(lens) if which != 2 else None, **before)
                    finally:
                        ops.attn_set_prefill_kernel(d, 1)
                        ops.attn_set_prefill_piece(d, 0)
                    _close(got, want, dtype, ("prompt", lens, which, piece, z is not None))
        assert ops.attn_tc05_timeouts(d) == 0
    c = case([1] * 5, [0, 63, 64, 200, 299])
    tok_pos, tok_seq, slots, first, start, end, table, kp, vp, rows = c
    for z in (sinks, None):
        want = statement(c, z)
        assert z is None or (want.float() - statement(c, None).float()).abs().max().item() > 0.05
        for chunk in (64, 128, 320):
            chunks = -(-320 // chunk)
            scratch = torch.full((ops.attn_decode_scratch_floats(5, H, d, chunks),), float("nan"), device="cuda")
            got = torch.full((5, H * d), float("nan"), dtype=dtype, device="cuda")
            ops.attn_decode_rows(*_cuda(rows, kp, vp, table, slots, end), scratch, got, H, G, d, scale, window, chunk, chunks,
                                 sinks=z.cuda() if z is not None else None)
            _close(got, want, dtype, ("decode", chunk, z is not None))
    assert ops.attn_wait_timeouts(d) == 0


@GPU
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,K,off", [(48, 4, 48), (21, 5, 3), (256, 2, 0), (10, 1, 4), (600, 4, 8)])
def test_filter_with_a_bias_on_its_inputs_against_its_statement(dtype, C, K, off):
    """The bias is part of the inputs, so it is absent before a sequence's start; kept inputs carry it."""
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    g = torch.Generator().manual_seed(15)
    for lens, starts, slots in (([9, 1, 2, 70, 3], [0, 5, 1, 0, 0], [2, 0, 4, 1, -1]), ([1, 1, 1], [0, 9, 3], [3, -1, 0])):
        tok_pos, tok_seq, *tabs = _tables(lens, starts, slots)
        T = sum(lens)
        rows = torch.randn(T, off + C + 5, generator=g).to(dtype)
        w, b, xb = torch.randn(C, K, generator=g), torch.randn(C, generator=g), torch.randn(C, generator=g)
        state = torch.randn(5, max(K - 1, 1), C, generator=g)
        for s, (st, slot) in enumerate(zip(starts, slots)):
            if st == 0 and slot >= 0:
                state[slot] = 0.0
        want, got, ws, gs = torch.zeros(T, C, dtype=dtype), torch.full((T, C), float("nan"), dtype=dtype, device="cuda"), state.clone(), state.cuda()
        one = max(lens) == 1
        R.causal_conv_silu(rows, off, C, w, b, ws, tok_seq, *tabs, len(lens), want, one_token=one, act=False, in_bias=xb)
        ops.causal_conv_silu(rows.cuda(), off, C, w.cuda(), b.cuda(), gs, tok_seq.cuda(), *_cuda(*tabs), len(lens), got, one_token=one,
                             act=False, in_bias=xb.cuda())
        _close(got, want, dtype, ("filter", lens))
        if K > 1:
            _close(gs, ws, torch.float32, ("kept inputs", lens))


def _recurrence_case(C, blocks, T, dtype, seed, y_cols):
    g = torch.Generator().manual_seed(seed)
    n = C // blocks
    lam = torch.linspace(-12.0, 2.0, C)[torch.randperm(C, generator=g)]
    return dict(u=torch.randn(T, C, generator=g).to(dtype), w=(torch.randn(blocks, 2 * n, n, generator=g) * n ** -0.5).to(dtype),
                br=torch.randn(C, generator=g), bi=torch.randn(C, generator=g), decay=-8.0 * torch.nn.functional.softplus(lam),
                y=torch.randn(T, y_cols, generator=g).to(dtype), yb=torch.randn(C, generator=g)), g


@GPU
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,blocks", [(48, 3), (21, 3), (256, 2), (10, 1), (2560, 10), (40, 40)])
def test_gated_recurrence_kernels_against_their_statements(dtype, C, blocks):
    """Prompts that end at, just before and just after the kernel's rounds, sequences that go on from a stored state, one token,
    a padding sequence; states of untouched slots stay; few long sequences (narrow CTAs) and many (wide ones).  Then steps of
    single rows, whose gates' products the kernel forms itself."""
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    n, y_off, z_off = C // blocks, 5, 3
    many = [2] * 600 if C == 48 else [5, 6]
    for lens, starts in (([64, 1, 63, 65, 2, 128, 130, 3], [0, 9, 4, 0, 0, 0, 77, 0]), (many, [0] * len(many))):
        T, ns = sum(lens), len(lens)
        slots = [s if s != 7 else -1 for s in range(ns)]
        _, tok_seq, *tabs = _tables(lens, starts, slots)
        c, g = _recurrence_case(C, blocks, T, dtype, 21, y_off + C + 2)
        gates = torch.zeros(T, 2 * C)
        R.head_linear(c["u"], n, 0, c["w"], gates, 2 * n, 0)
        got_gates = torch.full((T, 2 * C), float("nan"), device="cuda")
        ops.head_linear(c["u"].cuda(), n, 0, c["w"].cuda(), got_gates, 2 * n, 0)
        _close(got_gates, gates, torch.float32, "gates")                                # float32 results of either type's operands
        state = torch.randn(ns + 2, C, generator=g)
        for st, slot in zip(starts, slots):
            if st == 0 and slot >= 0:
                state[slot] = 0.0
        z = torch.zeros(T, z_off + C + 1, dtype=dtype)
        want, ws, got, gs = z.clone(), state.clone(), z.cuda(), state.cuda()
        R.gated_recurrence_scan(c["u"], gates.view(T, blocks, 2 * n), n, c["br"], c["bi"], c["decay"], c["y"], y_off, c["yb"], *tabs, ns,
                                ws, want, z_off, 0.7)
        ops.gated_recurrence_scan(c["u"].cuda(), gates.cuda().view(T, blocks, 2 * n), n, *_cuda(c["br"], c["bi"], c["decay"], c["y"]), y_off,
                                  c["yb"].cuda(), *_cuda(*tabs), ns, gs, got, z_off, 0.7)
        _close(got, want, dtype, ("scan", ns), f32=1e-5, bf16=1e-2)
        _close(gs, ws, torch.float32, ("states", ns), f32=1e-5)
        assert torch.equal(gs[ns:].cpu(), state[ns:]) and bool((got[:, :z_off] == 0).all()) and bool((got[:, z_off + C:] == 0).all())
    for T in (1, 8, 13):
        c, g = _recurrence_case(C, blocks, T, dtype, 23, y_off + C)
        tok_seq = torch.arange(T, dtype=torch.int32)
        slots = torch.randperm(T + 2, generator=g)[:T].to(torch.int32)
        if T > 1:
            slots[T // 2] = -1
        state = torch.randn(T + 2, C, generator=g)
        z = torch.zeros(T, z_off + C, dtype=dtype)
        want, ws, got, gs = z.clone(), state.clone(), z.cuda(), state.cuda()
        R.gated_recurrence_rows(c["u"], c["w"], c["br"], c["bi"], c["decay"], c["y"], y_off, c["yb"], tok_seq, slots, ws, want, z_off, 1.3)
        ops.gated_recurrence_rows(*_cuda(c["u"], c["w"], c["br"], c["bi"], c["decay"], c["y"]), y_off, c["yb"].cuda(), tok_seq.cuda(), slots.cuda(),
                                  gs, got, z_off, 1.3)
        _close(got, want, dtype, ("rows", T), f32=1e-5, bf16=1e-2)
        _close(gs, ws, torch.float32, ("states", T), f32=1e-5)


@GPU
def test_a_channel_that_remembers_thousands_of_tokens_keeps_its_last_bits():
    """Decays just below 1 over 4,096 tokens: an error of one sign in every step (a rounded to a float) would add up to 1e-4 of
    the state; and the same tokens in pieces of uneven sizes leave the same state."""
    from janis_b200.kernels import ops
    C, T = 64, 4096
    g = torch.Generator().manual_seed(4)
    u = torch.rand(T, C, generator=g) + 0.5
    decay = -torch.logspace(-6.0, -3.0, C)
    gates, zero, y = torch.zeros(T, 1, 2 * C), torch.zeros(C), torch.full((T, C), 3.0)
    a = torch.exp(0.5 * decay.double())
    S = torch.zeros(C, dtype=torch.float64)
    for t in range(T):
        S = a * S + torch.sqrt(-torch.expm1(decay.double())) * 0.5 * u[t].double()
    i32 = lambda *x: torch.tensor(x, dtype=torch.int32, device="cuda")
    states = []
    for cuts in ((0, T), (0, 1, 3, 700, 701, 3001, T)):
        st = torch.zeros(1, C, device="cuda")
        for lo, hi in zip(cuts, cuts[1:]):
            out = torch.zeros(hi - lo, C, device="cuda")
            ops.gated_recurrence_scan(u[lo:hi].cuda().contiguous(), gates[lo:hi].cuda().contiguous(), C, zero.cuda(), zero.cuda(), decay.cuda(),
                                      y[lo:hi].cuda().contiguous(), 0, None, i32(0), i32(0), i32(lo), i32(hi), 1, st, out)
        states.append(st[0].cpu().double())
        assert ((states[-1] - S).abs() / S).max().item() < 3e-6, cuts
    assert ((states[0] - states[1]).abs() / S).max().item() < 3e-6


@GPU
@pytest.mark.parametrize("dtype", DTYPES)
def test_gate_into_a_shared_row_and_clamped_gate_against_their_statements(dtype):
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    g = torch.Generator().manual_seed(8)
    for T, n, g_off, o_off, per, gated in ((19, 64, 16, 8, 1, True), (5, 21, 3, 5, 1, True), (7, 48, 8, 0, 16, True), (33, 40, 0, 8, 1, False)):
        x, rows = torch.randn(T, n, generator=g).to(dtype), torch.randn(T, g_off + n + 8 - (g_off + n) % 8, generator=g).to(dtype)
        z = torch.zeros(T, o_off + n + (8 - (o_off + n) % 8), dtype=dtype)
        want, got = z.clone(), z.cuda()
        R.gate_place(x, rows if gated else None, g_off, want, o_off, -0.6, per)
        ops.gate_place(x.cuda(), rows.cuda() if gated else None, g_off, got, o_off, -0.6, per)
        _close(got, want, dtype, ("place", n))
    for T, I in ((1, 8), (37, 40), (300, 168)):
        gu = (4.0 * torch.randn(T, 2 * I, generator=g)).to(dtype)
        want, got = torch.zeros(T, I, dtype=dtype), torch.full((T, I), float("nan"), dtype=dtype, device="cuda")
        extra = dict(limit=1.5, alpha=1.702, up_add=1.0)
        R.gated_act(gu, want, R.ACT_CLAMPED, **extra)
        ops.gated_act(gu.cuda(), got, ops.ACT_CLAMPED, **extra)
        _close(got, want, dtype, ("clamped", I))
    if dtype == torch.bfloat16:
        for M, N, K in ((1, 16, 64), (8, 96, 136), (16, 640, 320), (3, 32768, 64)):
            x, w = torch.randn(M, K, generator=g).to(dtype), (torch.randn(N, K, generator=g) * 2 * K ** -0.5).to(dtype)
            want, got = torch.zeros(M, N // 2, dtype=dtype), torch.full((M, N // 2), float("nan"), dtype=dtype, device="cuda")
            R.gemv_bf16(x, w, want, R.EPI_GATED_CLAMP, 1.2, alpha=1.702, up_add=1.0)
            ops.gemv_bf16(x.cuda(), w.cuda(), got, ops.EPI_GATED_CLAMP, 1.2, alpha=1.702, up_add=1.0)
            _close(got, want, dtype, ("product", N))


@GPU
@pytest.mark.parametrize("E,count,keep,top,shared", [(6, 3, 2, 2, 40), (4, 2, 1, 1, 0), (12, 4, 3, 4, 16), (8, 8, 3, 2, 0), (5, 1, 1, 3, 7), (64, 8, 2, 6, 24)])
def test_router_by_the_best_of_a_group_and_plain_experts_against_their_statements(E, count, keep, top, shared):
    from janis_b200.kernels import ops
    from tests import kernel_refs as R
    from tests.plain import larulorn_plain as P
    g = torch.Generator().manual_seed(6)
    T = 53
    z = 3.0 * torch.randn(T, E, generator=g)
    want, other = torch.zeros(T, E), torch.zeros(T, E)
    R.moe_route(z, None, E, count, keep, top, 1.0, False, want, softmax=True, group_best=True)
    got = torch.full((T, E), float("nan"), device="cuda")
    ops.moe_route(z.cuda(), None, E, count, keep, top, 1.0, False, got, softmax=True, group_best=True)
    assert torch.equal(got.cpu() != 0, want != 0)
    _close(got, want, torch.float32, "weights")
    idx, w = P.route(z.double(), top, {"count": count, "keep": keep})
    _close(got, torch.zeros(T, E, dtype=torch.float64).scatter_(1, idx, w), torch.float32, "weights of the plain model")
    if E == 64:
        R.moe_route(z, None, E, count, keep, top, 1.0, False, other, softmax=True)
        assert not torch.equal(other != 0, want != 0)                # the two largest together would keep other groups
    for dtype in DTYPES:
        for ff in (16, 13):
            x = torch.randn(T, E * ff + shared, generator=g).to(dtype)
            wx, gx = x.clone(), x.cuda()
            R.moe_relu2(wx, want, E, ff, shared)
            ops.moe_relu2(gx, got, E, ff, shared)
            _close(gx, wx, dtype, ("plain experts", ff))
            gated = torch.cat([want, torch.rand(T, 1, generator=g)], 1).contiguous()
            wx, gx = x.clone(), x.cuda()
            R.moe_relu2(wx, gated, E, ff, shared, True)
            ops.moe_relu2(gx, gated.cuda(), E, ff, shared, True)
            _close(gx, wx, dtype, ("with a gate on the shared one", ff))


# ---------------------------------------------------------------------------
# the engine against the plain model
# ---------------------------------------------------------------------------

@pytest.mark.parametrize("on,dtype", CASES)
def test_whole_prompts_and_first_tokens(engines, plain, on, dtype):
    for key in keys_for(on):
        eng, every = engines(key, dtype, on, max_tokens=2048)
        lens = [1, 2, 3, 70, 150] if on == "cuda" else [1, 2, 40]
        reqs = _requests(LAR[key]["vocab"], lens, 11)
        got = run_requests(eng, reqs, lens)
        for r, g_ in zip(reqs, got):
            assert_logits(g_, plain(key, every, r), dtype, f"{key} whole {len(r)}")


@pytest.mark.parametrize("on,dtype", CASES)
def test_prompts_of_unequal_lengths_then_decoded_together(engines, plain, on, dtype):
    """Batches one after another, so that slots, pages and states are used again; a request of one token beside long ones;
    decoding carries the recurrence and the filter over their stored states and the attention across page borders."""
    for key in keys_for(on):
        eng, every = engines(key, dtype, on, max_tokens=2048)
        if on == "cuda":
            lens, prompts = [260, 1, 140, 67, 200, 30], [120, 1, 60, 64, 63, 5]
        else:
            lens, prompts = [40, 1, 30, 12], [20, 1, 6, 9]
        reqs = _requests(LAR[key]["vocab"], lens, 23)
        got = run_requests(eng, reqs, prompts, max_live=3 if on == "cuda" else 2)
        for r, g_ in zip(reqs, got):
            assert_logits(g_, plain(key, every, r), dtype, f"{key} batch {len(r)}")


@pytest.mark.parametrize("on,dtype", CASES)
def test_a_request_alone_and_in_company_and_token_by_token(engines, plain, on, dtype):
    for key in keys_for(on)[:4]:
        eng, every = engines(key, dtype, on, max_tokens=2048)
        n = 90 if on == "cuda" else 25
        reqs = _requests(LAR[key]["vocab"], [n, 17, n // 2], 31)
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
        reqs = _requests(LAR[key]["vocab"], lens, 41)
        got = run_in_pieces(eng, reqs, chunk)
        for r, g_ in zip(reqs, got):
            assert_logits(g_, plain(key, every, r), dtype, f"{key} pieces of {chunk}, {len(r)} tokens")


@GPU
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_recorded_steps(engines, plain, dtype):
    for key in ("A", "C"):
        eng, every = engines(key, dtype, "cuda", max_tokens=2048)
        reqs = _requests(LAR[key]["vocab"], [330, 300], 51)
        got = run_requests(eng, reqs, [10, 3])
        for r, g_ in zip(reqs, got):
            assert_logits(g_, plain(key, every, r), dtype, f"{key} long decoding")


@GPU
def test_chosen_experts_in_the_serving_type(lar_dirs, plain):
    """Mixtures that choose, in bfloat16: close calls move single rows and, through the recurrence, some that follow; half of
    all rows stay within the rounding."""
    for key in ("A", "B", "C", "D"):
        eng = make_engine(lar_dirs[(key, False)], "bfloat16", "cuda", max_tokens=2048)
        try:
            reqs = _requests(LAR[key]["vocab"], [90] * 6, 55)
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
        V = LAR[key]["vocab"]
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


@GPU
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_first_token_far_back_reaches_the_end_through_attention_and_recurrence(tmp_path_factory, dtype):
    """One layer alone, flat attention weights: the first of 260 keys keeps a 260th of them; slow decays.  With the right
    branch's constant at 0 the recurrence must not reach the end, with the left one's the attention must not."""
    flat = _att(2, 1, 16, 16, 0.25, rot=8)
    for kind, mixer in (("attention", dict(flat, v_mix=True)), ("parallel", _par(flat, 32, 2, 4, 0.0, 1.0)), ("parallel", _par(flat, 32, 2, 4, 1.0, 0.0))):
        d = str(tmp_path_factory.mktemp("larulorn_far"))
        write_larulorn(d, _model(120, 64, 1e-6, 4.0, [(kind, mixer, None)]), 78, qk_gain=1.0)
        eng = make_engine(d, dtype, "cuda", max_tokens=1024)
        try:
            base = random_tokens(120, 260, 6)
            other = [(base[0] + 1) % 120] + base[1:]
            for n in (260, 200):
                a, b = (run_requests(eng, [r], [n])[0][-1] for r in (base, other))
                assert (a - b).abs().max().item() > (1e-5 if dtype == "float32" else 0.0), (kind, n)
        finally:
            eng.close()


def test_the_first_mixing_layers_values_and_not_anothers_are_mixed_in(lar_dirs):
    """The oracle with a planted mistake (the values of the layer before instead of the first one's; no mixing at all) differs
    from the oracle by far more than any tolerance here."""
    from tests.plain import larulorn_plain as P
    cfg, w = P.load_folder(lar_dirs[("C", False)])
    toks = random_tokens(cfg["vocab"], 30, 3)
    right = P.forward(cfg, w, toks)
    real = P.sink_attention

    def chained(y, w_, pre, m, first):
        out = real(y, w_, pre, m, chained.last)
        if m.get("v_mix"):
            chained.last = out[1]
        return out

    chained.last = None
    for planted in (chained, lambda y, w_, pre, m, first: real(y, w_, pre, m, None)):
        P.sink_attention = planted
        try:
            wrong = P.forward(cfg, w, toks)
        finally:
            P.sink_attention = real
        assert (wrong - right).abs().max().item() > 0.05 * right.abs().max().item()


def test_shared_products_are_the_branches_own(lar_dirs):
    """The parallel mixer's one input product and one output product against its branches run one by one (the plain kernel
    statements, float32), in a prompt step."""
    from janis_b200.parts.base import StepContext
    eng = make_engine(lar_dirs[("B", False)], "float32", "refs", max_tokens=512)
    fused = eng.model.blocks[2].mixer
    eng2 = make_engine(lar_dirs[("B", False)], "float32", "refs", max_tokens=512)
    apart = eng2.model.blocks[2].mixer
    cut_in = [apart.spans[k][0] for k in apart.branches] + [apart.w_in.shape[0]]
    cut_out = [apart.spans[k][1] for k in apart.branches] + [apart.w_out.shape[1]]
    for i, (m, names) in enumerate(zip(apart.branches.values(), (("w_qkv", "w_o"), ("w_in", "w_o")))):
        setattr(m, names[0], apart.w_in[cut_in[i]:cut_in[i + 1]].contiguous())
        setattr(m, names[1], apart.w_out[:, cut_out[i]:cut_out[i + 1]].contiguous())
    T, W = 11, LAR_B["width"]
    x = torch.randn(T, W, generator=torch.Generator().manual_seed(2))
    outs = []
    for e, mixer in ((eng, fused), (eng2, apart)):
        slot = e.alloc_slot()
        e.cache.reserve(slot, T)
        e.cache.sync()
        tok_pos, tok_seq, slots, first, start, end = _tables([T], [0], [slot])
        ctx = StepContext(rt=e.rt, ws=e.stepper.ws, mode="prefill", n_tok=T, n_seq=1, tokens=tok_pos, tok_pos=tok_pos, tok_seq=tok_seq,
                          seq_slot=slots, seq_start=start, seq_end=end, seq_first_row=first, len_bound=T)
        line = e.cache.line(2, True)
        if mixer is fused:
            outs.append(mixer.forward(x, ctx, line).clone())
        else:
            outs.append(sum(mixer.scales[k] * m.forward(x, ctx, mixer._own(line, k)).clone() for k, m in mixer.branches.items()))
    assert (outs[0] - outs[1]).abs().max().item() < 1e-5 * outs[1].abs().max().item()


@pytest.mark.parametrize("on,dtype", CASES)
def test_greedy_generation_through_the_engine(engines, plain, on, dtype):
    for key in ("A", "B"):
        eng, every = engines(key, dtype, on, max_tokens=2048)
        prompts = _requests(LAR[key]["vocab"], [33, 5, 70] if on == "cuda" else [9, 4], 61)
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
def test_trace_replay_and_command_line_as_a_user_runs_them(lar_dirs, plain, tmp_path):
    key, every = "A", False
    reqs = _requests(LAR[key]["vocab"], [40, 9], 71)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": reqs[0][:30], "want": [0, 29]}, {"id": "b", "tokens": reqs[1][:5], "want": [4]}], "end": []}]
    for i in range(10):
        ents = [{"id": "a", "tokens": [reqs[0][30 + i]], "want": [0]}]
        if 5 + i < 9:
            ents.append({"id": "b", "tokens": [reqs[1][5 + i]], "want": [0]})
        steps.append({"step": i + 1, "entries": ents, "end": ["b"] if 5 + i == 8 else (["a"] if i == 9 else [])})
    out = tmp_path / "out"
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", lar_dirs[(key, every)], "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(11)]
    import numpy as np
    V = LAR[key]["vocab"]
    wa, wb = plain(key, every, reqs[0]), plain(key, every, reqs[1])
    first = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(-1, V).copy())
    assert_logits(first, torch.stack([wa[0], wa[29], wb[4]]), "float32", "trace step 0")
    for i in range(10):
        got = torch.from_numpy(np.fromfile(out / f"{i + 1}.f32", dtype="<f4").reshape(-1, V).copy())
        want = [wa[30 + i]] + ([wb[5 + i]] if 5 + i < 9 else [])
        assert_logits(got, torch.stack(want), "float32", f"trace step {i + 1}")
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "janis"), "generate", "--model", lar_dirs[(key, every)], "--dtype", "float32",
                        "--ids", ",".join(map(str, reqs[1])), "--max-tokens", "4", "--temp", "0", "--stop", ""],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    seq = list(reqs[1])
    for _ in range(4):
        seq.append(int(plain(key, every, seq)[-1].argmax()))
    assert ",".join(map(str, seq[len(reqs[1]):])) in p.stdout.replace(" ", ""), p.stdout


def test_the_comparison_model_of_the_benchmark_builds_at_every_size():
    from janis_b200 import LarulornConfig, build_model
    from janis_b200.benchmark import larulorn_like, load_config
    for name in ("gemma2-2b", "gemma2-9b", "gemma2-27b"):
        gemma = load_config(name)
        raw = larulorn_like(gemma, 4)
        cfg = LarulornConfig.from_dict(raw)
        assert [l.type for l in cfg.layers] == ["parallel", "attention", "parallel", "attention"]
        _, _, model = build_model(raw)
        assert model.hidden == gemma["hidden_size"] and model.vocab == gemma["vocab_size"]
        assert all(n.shape for n in model.tensor_specs().values() if n.shape != ())


# three layers at sizes that reach the launch shapes, vector loads and library products the small models do not
LAR_WIDE = _model(2048, 1024, 1e-6, 0.75, [
    ("attention", _att(8, 2, 128, 128, 0.09, rot=64, base=100000.0, ramp=(8.0, 256, 32.0, 1.0), v_mix=True), _moe(8, 2, 512, (4, 2), shared=512)),
    ("parallel", _par(_att(8, 4, 128, 64, 0.09, rot=128, base=100000.0), 1280, 5, 4, 0.6, 0.8), _dense(2048, 3.0)),
    ("attention", _att(16, 2, 64, 128, 0.1, rot=64, base=5000.0, v_mix=True), _moe(8, 2, 512, (4, 2), shared=512))])


@GPU
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_three_layers_at_the_sizes_of_a_larger_model(tmp_path_factory, dtype):
    from tests.plain import larulorn_plain as P
    d = str(tmp_path_factory.mktemp("larulorn_wide"))
    write_larulorn(d, all_experts(LAR_WIDE) if dtype == "bfloat16" else LAR_WIDE, 91, gain=1.0, qk_gain=2.0, router_gain=6.0)
    cfg, w = P.load_folder(d)
    eng = make_engine(d, dtype, "cuda", max_tokens=4096)
    try:
        reqs = _requests(LAR_WIDE["vocab"], [560, 300, 40], 95)
        got = run_requests(eng, reqs, [520, 270, 3])
        for r, g_ in zip(reqs, got):
            assert_logits(g_, P.forward(cfg, w, r), dtype, f"wide {len(r)}")
    finally:
        eng.close()
