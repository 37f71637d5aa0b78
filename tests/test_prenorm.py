"""Pre-norm decoders (Seredra) on the CPU path: each mechanism, the step function, the cache, the engine and the loaders against the
plain restatement in tests/prenorm_oracle.py."""
import copy
import json
import math
import os
import subprocess
import urllib.request

import numpy as np
import pytest
import torch

import prenorm_checks as C
import prenorm_oracle as O
from rustral_b200.core.errors import SerializationError, ShapeMismatch
from rustral_b200.io import safetensors_io as st
from rustral_b200.models.config import preset
from rustral_b200.models.layered import AttentionSpec, LayeredConfig, MoESpec, RotarySpec, SelectiveSpec
from rustral_b200.models.registry import ARCHITECTURES
from rustral_b200.ops import (ScoreRule, Segments, attention_reference, gated_norm, head_prep_, residual_norm, rotary_table, rotate_halves, row_prep_,
                              selective_scan, short_conv, state_space)
from rustral_b200.ops import moe as moe_ops
from rustral_b200.ops.paged import paged_attention_rows
from rustral_b200.serve import PagedCache, ServingEngine
from rustral_b200.serve.kv_cache import CacheLayer
from rustral_b200.serve.model_runner import load_runner
from rustral_b200.serve.weights import InferenceWeights

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32 = torch.float32


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def table_of(rot, pos):
    spec = RotarySpec.from_json(rot, True)
    return rotary_table(pos, torch.tensor(spec.frequencies(), dtype=torch.float64), spec.magnitude)


# ---- mechanisms ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rot", [dict(dims=8, base=5000.0), dict(dims=2, base=100.0), dict(dims=16, base=2e4, scaling=dict(factor=3.0, original=512, fast=16.0, slow=1.0))],
                         ids=str)
def test_halves_turn_together(rot):
    spec = RotarySpec.from_json(rot, True)
    f, m = O.frequencies(rot)
    assert spec.half and spec.frequencies() == pytest.approx(f, rel=1e-12) and spec.magnitude == pytest.approx(m)
    assert RotarySpec.from_json(spec.to_json(), True) == spec and not RotarySpec.from_json(rot).half
    pos, x = torch.tensor([0, 1, 5, 77, 100000]), rnd(5, 3, rot["dims"] + 5)
    assert torch.allclose(rotate_halves(x, table_of(rot, pos)), O.rotate(x.double(), pos, rot).float(), atol=1e-5)


@pytest.mark.parametrize("dk,dims,keys", [(16, 8, True), (20, 12, False), (8, 8, True)])
def test_head_prep_with_halves_and_values_that_are_keys(dk, dims, keys):
    T, H, G = 6, 4, 2
    rot, pos = dict(dims=dims, base=300.0), torch.tensor([0, 3, 4, 50, 51, 9])
    p, gq, gk = rnd(T, (H + 2 * G) * dk + 3), rnd(dk, seed=1), rnd(dk, seed=2)
    q, k = p[:, :H * dk].clone(), p[:, H * dk:(H + G) * dk].clone()
    want_q = O.rotate(O.unit_rms(q.view(T, H, dk), 1e-3) * gq, pos, rot)
    want_k = O.rotate(O.unit_rms(k.view(T, G, dk), 1e-3) * gk, pos, rot)
    v = k if keys else p[:, (H + G) * dk:(H + 2 * G) * dk].clone()
    kc, vc, slots = torch.zeros(2, 4, G, dk), torch.zeros(2, 4, G, dk), torch.tensor([7, 0, -1, 2, 3, 5])
    head_prep_(p, H, G, dk, dk, q_gamma=gq, k_gamma=gk, eps=1e-3, rot=table_of(rot, pos), half=True, k_cache=kc, v_cache=vc, slots=slots, values_are_keys=keys)
    assert torch.allclose(p[:, :H * dk].view(T, H, dk), want_q, atol=1e-5) and torch.equal(p[:, (H + G) * dk:(H + 2 * G) * dk], v)
    keep = slots >= 0
    assert torch.allclose(kc.view(8, G, dk)[slots[keep]], want_k[keep], atol=1e-5) and torch.equal(vc.view(8, -1)[slots[keep]], v[keep])


def test_key_scale_and_columns():
    T, H, dk = 4, 3, 8
    rot, pos, p = dict(dims=6, base=50.0), torch.tensor([2, 0, 9, 33]), rnd(4, 60)
    q, k, rest = p[:, 30:54].clone(), p[:, 3:27].clone(), p[:, :3].clone()
    head_prep_(p, H, H, dk, dk, rot=table_of(rot, pos), half=True, k_scale=0.3, q_col=30, k_col=3)
    assert torch.allclose(p[:, 30:54], O.rotate(q.view(T, H, dk), pos, rot).reshape(T, -1), atol=1e-5) and torch.equal(p[:, :3], rest)
    assert torch.allclose(p[:, 3:27], 0.3 * O.rotate(k.view(T, H, dk), pos, rot).reshape(T, -1), atol=1e-5)
    with pytest.raises(ValueError):
        head_prep_(p, H, H, dk, dk, k_scale=0.3)


@pytest.mark.parametrize("every,coef", [(1, 0.5), (7, 0.3), (64, 2.0)])
def test_norm_over_the_row_and_temperature(every, coef):
    T, H, G, dk, dv = 5, 3, 2, 6, 5
    p, gq, gk = rnd(T, H * dk + G * (dk + dv)), rnd(H * dk, seed=1), rnd(G * dk, seed=2)
    pos = torch.tensor([0, every - 1, every, 2 * every - 2, 5 * every + 1]).clamp(min=0)
    t = O.temperature(pos, coef, every).float()[:, None]
    assert O.temperature([every - 2 if every > 1 else -1], coef, every)[0] == 1 and O.temperature([every - 1], coef, every)[0] == pytest.approx(1 + coef * math.log(2))
    want_q, want_k = O.unit_rms(p[:, :18], 1e-2) * gq * t, O.unit_rms(p[:, 18:30], 1e-2) * gk
    v, kc, vc, slots = p[:, 30:].clone(), torch.zeros(2, 4, G, dk), torch.zeros(2, 4, G, dv), torch.tensor([7, 0, -1, 2, 3])
    row_prep_(p, H, G, dk, dv, q_gamma=gq, k_gamma=gk, eps=1e-2, pos=pos, temp_coef=coef, temp_every=every, k_cache=kc, v_cache=vc, slots=slots)
    assert torch.allclose(p[:, :18], want_q, atol=1e-5) and torch.allclose(p[:, 18:30], want_k, atol=1e-5) and torch.equal(p[:, 30:], v)
    keep = slots >= 0
    assert torch.equal(kc.view(8, -1)[slots[keep]], p[keep, 18:30]) and torch.equal(vc.view(8, -1)[slots[keep]], v[keep])
    q = rnd(T, 18)
    want = O.unit_rms(q, 1e-2) * gq
    assert torch.allclose(row_prep_(q, H, 0, dk, dv, q_gamma=gq, eps=1e-2), want, atol=1e-5)                # no keys, no temperature


@pytest.mark.parametrize("cap,logs,scale", [(0.0, True, 1.0), (3.0, False, 0.4), (2.0, True, 1.7)])
def test_score_rule_with_cap_logarithmic_bias_and_output_scale(cap, logs, scale):
    q, k, v = rnd(23, 6, 8), rnd(23, 2, 8, seed=1), rnd(23, 2, 5, seed=2)
    r1, r2 = (rnd(6, seed=3).abs(), rnd(6, seed=4).abs()) if logs else (None, None)
    rule = ScoreRule(softcap=cap, log_amount=r1, log_rate=r2, out_scale=scale)
    want = scale * O.attend(q, k, v, 0.9, cap, r1, r2)
    assert not rule.plain and torch.allclose(attention_reference(q[None], k[None], v[None], True, 0.9, rule=rule)[0], want, atol=1e-5)
    last = attention_reference(q[None, -4:], k[None], v[None], True, 0.9, rule=rule)[0]                     # queries at the end of more keys
    assert torch.allclose(last, want[-4:], atol=1e-5)
    kc, vc, bt = torch.full((5, 8, 2, 8), 1e4), torch.full((5, 8, 2, 5), 1e4), torch.tensor([[4, 0, 3]], dtype=torch.int32)
    for t in range(23):
        kc[bt[0, t // 8], t % 8], vc[bt[0, t // 8], t % 8] = k[t], v[t]
    got = paged_attention_rows(q.reshape(23, -1), kc, vc, bt, torch.zeros(23, dtype=torch.int32), torch.arange(23), 0.9, rule)
    assert torch.allclose(got.view(23, 6, 5), want, atol=1e-5)


def test_a_far_key_that_stands_out_pays_the_logarithmic_bias_only():
    """Distance 46 costs r1 ln(1 + 46 r2): a score of 9 above the others beats 2 ln 24 but not 4 ln 24."""
    q, k, v = C.standout_case(47, 1, 48, 2, 1, 16, 4)
    q, k = 0 * q, 0 * k
    q[47, :, 0], k[1, 0, 0] = 3.0, 3.0
    for r1, wins in ((2.0, True), (4.0, False)):
        o = attention_reference(q[None], k[None], v[None], True, 1.0, rule=ScoreRule(log_amount=torch.full((2,), r1), log_rate=torch.full((2,), 0.5)))[0]
        w = math.exp(9 - r1 * math.log(24)) / (math.exp(9 - r1 * math.log(24)) + sum(math.exp(-r1 * math.log(1 + 0.5 * d)) for d in range(48) if d != 46))
        assert (w > 0.5) == wins
        other = sum(math.exp(-r1 * math.log(1 + 0.5 * (47 - j))) * v[j, 0] for j in range(48) if j != 1) / sum(math.exp(-r1 * math.log(1 + 0.5 * (47 - j))) for j in range(48) if j != 1)
        assert torch.allclose(o[47, 0], w * v[1, 0] + (1 - w) * other, atol=1e-4)


def segments_case(T=40):
    """Rows of five sequences: new ones, continued ones, single rows."""
    return [(0, 13, 2, 0), (13, 1, 0, 9), (14, 5, 1, 3), (19, 2, 3, 0), (21, T - 21, 5, 8)]


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_convolution_without_activation(taps):
    x, w, state = rnd(40, 6), rnd(6, taps, seed=1), rnd(6, taps - 1, 6, seed=2)
    before, segs = state.clone(), segments_case()
    got = short_conv(x, w, None, state, Segments.of(segs, "cpu"), silu=False)
    for first, n, slot, start in segs:
        past = before[slot] if start else torch.zeros(taps - 1, 6)
        full = torch.cat([past, x[first:first + n]])
        assert torch.allclose(got[first:first + n], O.causal_conv(full, w)[taps - 1:], atol=1e-5)
        assert torch.equal(state[slot], full[n:])


@pytest.mark.parametrize("inner,n", [(6, 4), (5, 3), (7, 1)])
def test_selective_scan_over_segments(inner, n):
    T, segs = 40, segments_case()
    x, dt, B, Cc, z = rnd(T, inner), rnd(T, inner, seed=1), rnd(T, n, seed=2), rnd(T, n, seed=3), rnd(T, inner, seed=4)
    A, D, bias = -rnd(inner, n, seed=5).abs(), rnd(inner, seed=6), rnd(inner, seed=7) - 2
    state = rnd(6, inner, (n + 3) // 4 * 4, seed=8)
    before = state.clone()
    got = selective_scan(x, dt, B, Cc, z, A=A, D=D, dt_bias=bias, state=state, seg=Segments.of(segs, "cpu"), scale=0.6)
    step = O.softplus(dt + bias)
    for first, m, slot, start in segs:
        rows = slice(first, first + m)
        S = before[slot, :, :n].clone() if start else torch.zeros(inner, n)
        for t in range(first, first + m):
            S = torch.exp(step[t][:, None] * A) * S + (step[t] * x[t])[:, None] * B[t][None, :]
            assert torch.allclose(got[t], 0.6 * (S @ Cc[t] + D * x[t]) * O.silu(z[t]), atol=1e-4)
        assert torch.allclose(state[slot, :, :n], S, atol=1e-4)
        if start == 0:
            want = 0.6 * O.scan(x[rows], step[rows], B[rows], Cc[rows], A, D) * O.silu(z[rows])
            assert torch.allclose(got[rows], want, atol=1e-4)


def test_fixed_decay_recurrence():
    T, H, n, dv = 30, 3, 4, 5
    v, k, q, decay = rnd(T, H, dv), rnd(T, H, n, seed=1), rnd(T, H, n, seed=2), torch.tensor([1.0, 0.5, 0.99])
    packed = torch.cat([v.reshape(T, -1), k.reshape(T, -1), q.reshape(T, -1)], 1)
    state = torch.full((2, H, n, 8), 1e4)
    a = state_space(packed[:17], decay=decay, state=state, heads=H, groups=H, vdim=dv, n=n, seg=Segments.of([(0, 17, 1, 0)], "cpu"))
    b = state_space(packed[17:], decay=decay, state=state, heads=H, groups=H, vdim=dv, n=n, seg=Segments.of([(0, 13, 1, 17)], "cpu"))
    assert torch.allclose(torch.cat([a, b]).view(T, H, dv), O.retain(q, k, v, decay), atol=1e-4)
    y, g = rnd(6, 12), rnd(6, 12, seed=1)
    assert torch.allclose(gated_norm(y, g, None, 3, 1e-3, gate_first=False), O.unit_rms(y.view(6, 3, 4), 1e-3).reshape(6, 12) * O.silu(g), atol=1e-5)


def test_residual_add_with_a_norm_behind():
    x, y, g, h = rnd(5, 16), rnd(5, 16, seed=1), torch.full((16,), 0.7), torch.empty(5, 16)
    x1 = x.clone()
    residual_norm(y, None, None, 1e-2, True, x=x1, h=h, next_gamma=g)
    assert torch.equal(x1, x + y) and torch.allclose(h, O.scalar_norm(x + y, torch.tensor(0.7), 1e-2), atol=1e-6)
    rows, slots = rnd(20, 16, seed=4), torch.tensor([3, 7, 0, 19, 5, 5, 2, 1, 9, 8], dtype=torch.int32)
    x2 = x.clone()
    residual_norm(rows, None, None, 1e-2, True, x=x2, h=h, next_gamma=g, routed=(slots, None))
    assert torch.allclose(x2, x + rows[slots.long()].view(5, 2, 16).sum(1), atol=1e-6)
    x3 = x.clone()
    assert residual_norm(y, None, None, 1e-2, True, x=x3) is x3 and torch.equal(x3, x + y)


@pytest.mark.parametrize("E,k", [(6, 2), (5, 5), (1, 1)])
def test_expert_weights_multiply_the_input(E, k):
    T, d, ff = 9, 8, 16
    x, router = rnd(T, d), rnd(E, d, seed=1)
    w = {f"e{e}.{n}": rnd(*s, seed=10 * e + i) for e in range(E) for i, (n, s) in enumerate((("gate", (ff, d)), ("up", (ff, d)), ("down", (d, ff))))}
    w["router"] = router
    want = O.routed_ff(x, w, "", {"router": {"top": k}})
    idx, ws = moe_ops.route_sigmoid(x @ router.T, k)
    for t in range(T):
        i, s = O.choose(x[t] @ router.T, k)
        assert idx[t].tolist() == i and torch.allclose(ws[t], s, atol=1e-6)
    pl = moe_ops.plan(idx, E)
    w1 = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(E)])
    gu = moe_ops.grouped_gemm(moe_ops.scatter_tokens(x, pl), w1, pl)
    y = moe_ops.grouped_gemm(moe_ops.swiglu_rows(gu, pl, weights=ws), torch.stack([w[f"e{e}.down"] for e in range(E)]), pl)
    assert torch.allclose(y[pl.slot_pos.long()].view(T, k, d).sum(1), want, atol=1e-4)


# ---- cache ----------------------------------------------------------------------------------------------------------
def test_layers_without_keys_of_their_own():
    c = PagedCache(4, 8, dtype=F32, layers=[CacheLayer(2, 4, 3), CacheLayer(state=(("s", (5,), None),)), CacheLayer(2, 4, 3, kv_of=0)], num_slots=2)
    assert c.k[2] is c.k[0] and c.v[2] is c.v[0] and c.k[1] is None and c.memory_bytes() == 4 * (4 * 8 * 2 * 7 + 2 * 5)
    r = C.runner(C.CONFIGS["varied"], C.weights(C.CONFIGS["varied"]))
    assert r.cache.k[3] is r.cache.k[1] and r.cache.v[6] is r.cache.v[1] and r.cache.k[2] is None and r.body.lent == {1}
    assert r.cache.state[1]["conv"].shape[2] == 6 * 16 + 2 * 56 and r.cache.state[3]["conv"].shape == (4, 1, 64) and r.cache.state[0]["state"].dtype == F32


@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_prefill_portions_and_decoding_agree_with_the_plain_model(name):
    C.check_prefill_portions_and_decode(name, "cpu", F32, 70 if name not in ("wide", "dense") else 40)


@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_mixed_batches_with_reused_pages(name):
    C.check_mixed_batch_with_reused_pages(name, "cpu", F32)


def test_long_decoding():
    C.check_long_decoding("varied", "cpu", F32, 150)


def test_first_tokens_of_a_sequence():
    cfg = C.CONFIGS["varied"]
    w = C.weights(cfg, 8)
    for n in (1, 2, 3):
        toks = C.tokens(cfg, n, n)
        C.assert_logits(C.feed(C.runner(cfg, w), 0, toks, []), C.reference(cfg, w, toks), F32, n)


@pytest.mark.parametrize("block_size", [1, 4, 64])
def test_other_page_sizes(block_size):
    cfg = C.CONFIGS["varied"]
    w = C.weights(cfg, 9)
    toks = C.tokens(cfg, 50, 3)
    r = C.runner(cfg, w, blocks=128, block_size=block_size)
    C.assert_logits(C.feed(r, 0, toks, [5, 7, 33, 34, 35]), C.reference(cfg, w, toks), F32, block_size)


def _mixer(i, *path, **new):
    def change(c, w):
        m = c["layers"][i]["mixer"]
        for p in path:
            m = m[p]
        m.update(new)
    return change


MISTAKES = {
    "cap": _mixer(0, "left", softcap=5.0),
    "no cap": lambda c, w: c["layers"][0]["mixer"]["left"].pop("softcap"),
    "scale": _mixer(1, scale=0.38),
    "left scale": _mixer(0, left_scale=1.25),
    "right scale": _mixer(5, right_scale=1.8),
    "rotated dims": _mixer(0, "left", "rot", dims=14),
    "base": _mixer(2, "rot", base=400.0),
    "yarn": lambda c, w: c["layers"][0]["mixer"]["left"]["rot"].pop("scaling"),
    "yarn factor": _mixer(0, "left", "rot", "scaling", factor=5.0),
    "yarn ramp": _mixer(0, "left", "rot", "scaling", slow=0.02),
    "a second pair": _mixer(5, "left", "rot", dims=4),
    "temperature": _mixer(1, "q_temp", coef=0.5),
    "temperature step": _mixer(6, "q_temp", every=21),
    "no temperature": lambda c, w: c["layers"][6]["mixer"].pop("q_temp"),
    "decay": _mixer(2, decay=[0.8, 0.97, 0.99]),
    "decay of one": _mixer(4, decay=[0.999, 0.5]),
    "embedding scale": lambda c, w: c["embedding"].update(scale=2.6),
    "eps": lambda c, w: c["norm"].update(eps=1e-2),
    "norm in front": lambda c, w: w["l2.norm1"].fill_(1),
    "norm in front of a feed-forward": lambda c, w: w["l0.norm2"].fill_(1),
    "final norm": lambda c, w: w["final.norm"].mul_(1.1),
    "query norm": lambda c, w: w["l1.mix.q.norm"].fill_(1.6),
    "key norm": lambda c, w: w["l0.mix.left.k.norm"].fill_(1.6),
    "query bias": lambda c, w: w["l3.mix.q.b"].zero_(),
    "key bias": lambda c, w: w["l1.mix.k.b"].zero_(),
    "value bias": lambda c, w: w["l1.mix.v.b"].zero_(),
    "output bias": lambda c, w: w["l6.mix.o.b"].zero_(),
    "convolution of the keys": lambda c, w: w["l1.mix.k.conv"][:, 0].zero_(),
    "convolution of the values": lambda c, w: w.update({"l1.mix.v.conv": w["l1.mix.v.conv"].flip(1)}),
    "convolution of the queries": lambda c, w: w.update({"l3.mix.q.conv": w["l3.mix.q.conv"].flip(1)}),
    "bias amount": lambda c, w: w["l6.mix.r1"].mul_(0.8),
    "bias rate": lambda c, w: w["l3.mix.r2"].mul_(0.7),
    "scan convolution bias": lambda c, w: w["l0.mix.right.conv.b"].zero_(),
    "step bias": lambda c, w: w["l5.mix.right.dt.b"].zero_(),
    "skip": lambda c, w: w["l0.mix.right.D"].zero_(),
    "state decay": lambda c, w: w["l0.mix.right.A_log"].zero_(),
    "retention gate": lambda c, w: w["l4.mix.g"].neg_(),
    "keys of another layer": lambda c, w: c["layers"][6]["mixer"].pop("kv_from") and w.update({f"l6.mix.{n}": w[f"l1.mix.{n}"].flip(0) for n in (
        "k", "v", "k.b", "v.b", "k.norm", "k.conv", "v.conv")}),
}


def _patches():
    plain_rotate, plain_attend, plain_choose = O.rotate, O.attend, O.choose

    def neighbours(x, positions, rot):
        y, n = x.clone(), rot["dims"]
        y[..., :n] = torch.cat([x[..., 0:n:2], x[..., 1:n:2]], -1)
        z = plain_rotate(y, positions, rot)
        out = z.clone()
        out[..., 0:n:2], out[..., 1:n:2] = z[..., :n // 2], z[..., n // 2:n]
        return out

    def values_with_norm(x, w, p, m, eps):
        T, G, n = x.shape[0], m["kv_heads"], m["dim"]
        k = plain_rotate(O.unit_rms((x @ w[p + "k"].T).view(T, G, n), eps) * w[p + "k.norm"], torch.arange(T), m["rot"])
        q = plain_rotate(O.unit_rms((x @ w[p + "q"].T).view(T, -1, n), eps) * w[p + "q.norm"], torch.arange(T), m["rot"])
        return plain_attend(q, k, k, m["scale"], m.get("softcap") or 0.0).reshape(T, -1) @ w[p + "o"].T

    def output_weights(x, w, p, f):
        z, out = x @ w[p + "router"].T, torch.zeros_like(x)
        for t in range(x.shape[0]):
            for e, we in zip(*plain_choose(z[t], f["router"]["top"])):
                out[t] += we * O.expert(x[t], w, f"{p}e{e}.")
        return out

    def renormed(z, top):
        i, s = plain_choose(z, top)
        return i, s / s.sum()
    return {"pairing": ("rotate", neighbours), "values behind the norm": ("key_value_attention", values_with_norm),
            "linear bias": ("attend", lambda q, k, v, s, cap=0.0, r1=None, r2=None: plain_attend(q, k, v, s, cap, None if r1 is None else 0.9 * r1, r2)),
            "weights on the output": ("routed_ff", output_weights), "renormed weights": ("choose", renormed),
            "one step late": ("temperature", lambda pos, coef, every: torch.tensor([1 + coef * math.log(int(p) // every + 1) for p in pos], dtype=torch.float64)),
            "no norm of the retention's output": ("retain", lambda q, k, v, d: 0.5 * v),
            "relu": ("relu2_ff", lambda x, w, p: torch.relu(x @ w[p + "up"].T) @ w[p + "down"].T)}


@pytest.mark.parametrize("mistake", [*MISTAKES, *_patches()])
def test_the_comparison_notices_a_mistake(mistake, monkeypatch):
    """The plain model with one thing changed must not agree: the checks above would see such a fault."""
    cfg = C.CONFIGS["varied"]
    w = {k: v.clone() for k, v in C.weights(cfg).items()}
    toks = C.tokens(cfg, 60)
    got = C.feed(C.runner(cfg, w), 0, toks, [])
    bad = copy.deepcopy(cfg)
    if mistake in MISTAKES:
        MISTAKES[mistake](bad, w)
    else:
        name, fn = _patches()[mistake]
        monkeypatch.setattr(O, name, fn)
    with pytest.raises(AssertionError):
        C.assert_logits(got, C.reference(bad, w, toks), F32)


# ---- the engine -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("prefill_chunk", [0, 8, 2048])
def test_greedy_generation_through_the_engine(prefill_chunk):
    cfg = C.CONFIGS["varied"]
    w = C.weights(cfg, 6)
    r = C.runner(cfg, w, blocks=40, slots=3)
    C.poison(r)
    eng = ServingEngine(r, max_batch_size=3, prefill_chunk=prefill_chunk)
    prompts = [C.tokens(cfg, n, 20 + n) for n in (5, 19, 33, 1)]
    ids = [eng.submit(p, 5) for p in prompts]
    eng.run_to_completion()
    wd = {k: v.double() for k, v in w.items()}
    for p, rid in zip(prompts, ids):
        assert eng.scheduler.get(rid).generated == O.greedy(cfg, wd, p, 5)
    assert r.cache.free_blocks == 40 and r.cache.free_slots == 3


def test_engine_recomputes_a_request_that_was_paused_for_memory():
    cfg = C.CONFIGS["single"]
    w = C.weights(cfg, 7)
    eng = ServingEngine(C.runner(cfg, w, blocks=6, block_size=4), max_batch_size=4, prefill_chunk=4)
    prompts = [C.tokens(cfg, n, 40 + n) for n in (7, 6, 5)]
    ids = [eng.submit(p, 9) for p in prompts]
    eng.run_to_completion()
    wd = {k: v.double() for k, v in w.items()}
    assert eng.scheduler.stats.preempted > 0
    for p, rid in zip(prompts, ids):
        assert eng.scheduler.get(rid).generated == O.greedy(cfg, wd, p, 9)


# ---- configuration, loading, command line ---------------------------------------------------------------------------
def save_model(folder, cfg, w):
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(st.serialize(w))


def test_config_round_trip_and_registry():
    for cfg in C.CONFIGS.values():
        lc = LayeredConfig.from_json(cfg)
        assert LayeredConfig.from_json(lc.to_json()) == lc
        assert lc.num_parameters() == sum(int(np.prod(s)) for s in lc.tensor_shapes().values())
    lc = LayeredConfig.from_json(C.CONFIGS["varied"])
    shapes = lc.tensor_shapes()
    assert lc.embed_scale == 2.5 and lc.norm_eps == 1e-3 and lc.layers[3].mlp is None and shapes["l0.norm1"] == () and "l3.norm2" not in shapes
    assert {n for n in shapes if n.startswith("l3.mix.")} == {"l3.mix." + n for n in ("q", "q.b", "q.conv", "q.norm", "r1", "r2", "o", "o.b")}
    a, left = lc.layers[1].mixer, lc.layers[0].mixer.left
    assert isinstance(a, AttentionSpec) and a.norm_over == "all" and a.log_bias and a.out_bias and (a.temp_coef, a.temp_every, a.conv) == (0.6, 7, 3) and a.rot is None
    assert left.values_are_keys and left.rot.half and left.softcap == 4.0 and not left.bias and "l0.mix.left.v" not in shapes
    assert lc.layers[0].mixer.right == SelectiveSpec(40, 12, 6, 4) and lc.layers[0].mixer.scales == (1.3, 0.7) and lc.layers[2].mixer.decay == (0.8, 0.97, 0.999)
    assert lc.layers[0].mlp == MoESpec(24, 8, 2, score="sigmoid", renorm=False, weigh="input")
    assert "Seredra" in ARCHITECTURES and ARCHITECTURES["Seredra"].float32
    p = preset("seredra-test")
    assert p.n_layer == 4 and p.layers[3].mixer.kv_from == 1 and preset("seredra-moe", n_layer=7).n_layer == 7
    bads = [lambda c: c["layers"][0].update(type="delta"), lambda c: c["layers"][0]["mlp"].update(kind="swiglu"), lambda c: c["layers"][3]["mixer"].update(kv_from=4),
            lambda c: c["layers"][3]["mixer"].update(kv_from=3), lambda c: c["layers"][3]["mixer"].update(kv_from=2), lambda c: c["layers"][6]["mixer"].update(kv_from=3),
            lambda c: c["layers"][3]["mixer"].update(vdim=32), lambda c: c["layers"][0]["mixer"]["left"].update(vdim=16), lambda c: c["layers"][2]["mixer"].update(decay=[0.5, 0.5]),
            lambda c: c["layers"][2]["mixer"].update(decay=[0.5, 0.5, 1.5]), lambda c: c["layers"][2]["mixer"]["rot"].update(dims=18), lambda c: c["layers"][1]["mixer"].update(kv_heads=4),
            lambda c: c["layers"][0]["mixer"]["right"].update(state=0), lambda c: c["layers"][0]["mlp"]["router"].update(top=9)]
    for bad in bads:
        c = copy.deepcopy(C.CONFIGS["varied"])
        bad(c)
        with pytest.raises(ValueError):
            LayeredConfig.from_json(c)


def test_random_weights_and_preset_run():
    from rustral_b200.serve import ModelRunner
    cfg = preset("seredra-test")
    out = ServingEngine(ModelRunner(cfg, device="cpu", num_blocks=16)).generate([1, 2, 3], 3)
    assert len(out) == 3 and all(0 <= t < cfg.vocab_size for t in out)


def test_loading_is_strict(tmp_path):
    cfg = C.CONFIGS["varied"]
    lc, w = LayeredConfig.from_json(cfg), C.weights(cfg)
    for gone in ("l1.mix.k.conv", "l0.norm1", "l6.mix.o.b", "l0.mix.right.A_log", "l3.mix.r2", "head"):
        with pytest.raises(SerializationError):
            InferenceWeights.layered(lc, "cpu", None, {k: v for k, v in w.items() if k != gone})
    with pytest.raises(SerializationError):
        InferenceWeights.layered(lc, "cpu", None, {**w, "l3.mix.k": w["l1.mix.k"]})
    with pytest.raises(ShapeMismatch):
        InferenceWeights.layered(lc, "cpu", None, {**w, "l0.mix.right.x": w["l0.mix.right.x"][:-1]})
    save_model(tmp_path, cfg, {**w, "l3.norm2": w["l2.norm2"]})                  # a norm that nothing reads
    r = load_runner(str(tmp_path), device="cpu")
    toks = C.tokens(cfg, 30)
    C.assert_logits(C.feed(r, 0, toks, [11]), C.reference(cfg, w, toks), F32)


def test_trace_replay_program(tmp_path):
    cfg = C.CONFIGS["varied"]
    w = C.weights(cfg, 11)
    save_model(tmp_path, cfg, w)
    reqs = {f"r{i}": C.tokens(cfg, n, i) for i, n in enumerate((40, 21, 9))}
    want = {k: C.reference(cfg, w, t) for k, t in reqs.items()}
    plan = [([("r0", 17, [0, 16]), ("r1", 1, [])], []), ([("r1", 19, [18, 3]), ("r0", 1, [0]), ("r2", 2, [1])], []),
            ([("r0", 1, [0]), ("r1", 1, [0])], ["r1"]), ([("r2", 7, [6, 0]), ("r0", 21, [20])], ["r0", "r2"])]
    steps, expect, at = [], {}, {k: 0 for k in reqs}
    for i, (entries, end) in enumerate(plan):
        rows, ents = [], []
        for rid, n, places in entries:
            ents.append({"id": rid, "tokens": reqs[rid][at[rid]:at[rid] + n], "want": places})
            rows += [want[rid][at[rid] + p] for p in places]
            at[rid] += n
        expect[i] = torch.stack(rows)
        steps.append({"step": i, "entries": ents, "end": end})
    out = tmp_path / "out"
    out.mkdir()
    res = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out),
                          "--max-tokens", "128", "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                         capture_output=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    for i, x in expect.items():
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"])
        assert got.shape == x.shape
        C.assert_logits(got, x, F32, i)


def test_server_command_line_serves_a_model_folder(tmp_path):
    from rustral_b200.serve.http_server import build_state, parse_args, start_background
    cfg = C.CONFIGS["single"]
    w = C.weights(cfg, 12)
    save_model(tmp_path, cfg, w)
    state = build_state(parse_args(["--model", str(tmp_path), "--blocks", "32", "--max-batch", "4"]))
    httpd, _ = start_background(state)
    try:
        prompt = C.tokens(cfg, 9, 5)
        req = urllib.request.Request(f"http://127.0.0.1:{httpd.server_address[1]}/v1/generate",
                                     json.dumps({"prompt": prompt, "max_tokens": 5}).encode())
        assert json.load(urllib.request.urlopen(req))["tokens"] == O.greedy(cfg, {k: v.double() for k, v in w.items()}, prompt, 5)
    finally:
        httpd.shutdown()
        state.shutdown()
