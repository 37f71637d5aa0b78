"""Looped decoders (Bikilix) on the CPU path: each mechanism, the step function, the cache, the engine and the loaders against the plain
restatement in tests/looped_oracle.py."""
import copy
import json
import math
import os
import subprocess
import urllib.request

import numpy as np
import pytest
import torch

import looped_checks as C
import looped_oracle as O
from rustral_b200.core.errors import SerializationError, ShapeMismatch
from rustral_b200.io import safetensors_io as st
from rustral_b200.models.config import preset
from rustral_b200.models.layered import LayeredConfig, MoESpec, RotarySpec
from rustral_b200.models.registry import ARCHITECTURES
from rustral_b200.ops import (ScoreRule, act_reference, attention_reference, embedding_residual, gemm, head_prep_, head_product, latent_decode,
                              latent_prep_, linear, residual_norm, rotary_table, rotate_pairs_)
from rustral_b200.ops.attention import prompt_attention_split
from rustral_b200.ops.moe import route_sigmoid, swiglu_rows
from rustral_b200.serve import PagedCache, ServingEngine
from rustral_b200.serve.kv_cache import CacheLayer
from rustral_b200.serve.model_runner import load_runner
from rustral_b200.serve.weights import InferenceWeights

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32 = torch.float32


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


ROTS = [dict(dims=8, base=5000.0), dict(dims=2, base=100.0), dict(dims=32, base=1e6, scaling=dict(factor=8.0, original=64, fast=16.0, slow=1.0)),
        dict(dims=16, base=2e4, scaling=dict(factor=3.0, original=4096, fast=32.0, slow=1.0)),
        dict(dims=12, base=50.0, scaling=dict(factor=40.0, original=30, fast=1.0, slow=0.5)),      # the ramp has no width
        dict(dims=6, base=1e4, scaling=dict(factor=1.0, original=128, fast=8.0, slow=1.0))]


def table_of(rot, pos):
    spec = RotarySpec.from_json(rot)
    return rotary_table(pos, torch.tensor(spec.frequencies(), dtype=torch.float64), spec.magnitude)


# ---- mechanisms ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rot", ROTS, ids=str)
def test_rotary_positions(rot):
    spec = RotarySpec.from_json(rot)
    f, m = O.frequencies(rot)
    assert spec.frequencies() == pytest.approx(f, rel=1e-12) and spec.magnitude == pytest.approx(m) and RotarySpec.from_json(spec.to_json()) == spec
    pos = torch.tensor([0, 1, 5, 77, 100000])
    x = rnd(5, 3, rot["dims"] + 5)
    want = O.rotate(x.double(), pos, rot).float()
    x2 = torch.zeros(5, 3 * (rot["dims"] + 9))
    x2.view(5, 3, -1)[..., 4:] = x                                            # the rotated part starts at column 4 of a head
    rotate_pairs_(x2, 3, rot["dims"] + 9, 4, table_of(rot, pos))
    assert torch.allclose(x2.view(5, 3, -1)[..., 4:], want, atol=1e-5) and float(x2.view(5, 3, -1)[..., :4].abs().max()) == 0


def test_yarn_slows_the_slow_pairs_only():
    s = RotarySpec(16, 2e4, 4.0, 512, 16.0, 1.0, True)
    plain = RotarySpec(16, 2e4).frequencies()
    ratio = [a / b for a, b in zip(s.frequencies(), plain)]
    turns = [512 * f / (2 * math.pi) for f in plain]
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(0.25) and ratio == sorted(ratio, reverse=True)
    assert all(r == 1.0 for r, t in zip(ratio, turns) if t >= 2 * 16) and all(r == pytest.approx(0.25) for r, t in zip(ratio, turns) if t <= 0.2)
    assert s.magnitude == pytest.approx(1 + 0.1 * math.log(4.0))
    for bad in (dict(dims=5, base=10.0), dict(dims=4, base=1.0), dict(dims=4, base=10.0, scaled=True, original=0)):
        with pytest.raises(ValueError):
            RotarySpec(**bad)


def test_scores_depend_on_the_distance_only():
    rot = ROTS[0]
    q, k = rnd(1, 1, 8), rnd(1, 1, 8, seed=1)
    dot = [float((O.rotate(q, torch.tensor([a]), rot) * O.rotate(k, torch.tensor([b]), rot)).sum()) for a, b in ((9, 2), (107, 100), (7, 0))]
    assert dot[0] == pytest.approx(dot[1], abs=1e-4) and dot[0] == pytest.approx(dot[2], abs=1e-4)


@pytest.mark.parametrize("dk,dv,dims", [(16, 8, 8), (20, 12, 6), (8, 8, 8)])
def test_head_prep_rotates_and_appends(dk, dv, dims):
    T, H, G = 6, 4, 2
    rot = dict(dims=dims, base=300.0)
    pos = torch.tensor([0, 3, 4, 50, 51, 9])
    p = rnd(T, H * dk + G * (dk + dv) + 3)
    want_q = O.rotate(p[:, :H * dk].reshape(T, H, dk), pos, rot)
    want_k = O.rotate(p[:, H * dk:(H + G) * dk].reshape(T, G, dk), pos, rot)
    v, rest = p[:, (H + G) * dk:(H + G) * dk + G * dv].clone(), p[:, -3:].clone()
    kc, vc = torch.zeros(2, 4, G, dk), torch.zeros(2, 4, G, dv)
    slots = torch.tensor([7, 0, -1, 2, 3, 5])
    head_prep_(p, H, G, dk, dv, k_cache=kc, v_cache=vc, slots=slots, rot=table_of(rot, pos))
    assert torch.allclose(p[:, :H * dk].view(T, H, dk), want_q, atol=1e-5) and torch.equal(p[:, -3:], rest)
    keep = slots >= 0
    assert torch.allclose(kc.view(8, G, dk)[slots[keep]], want_k[keep], atol=1e-5)
    assert torch.equal(vc.view(8, G * dv)[slots[keep]], v[keep]) and float(kc.view(8, -1)[[1, 4, 6]].abs().max()) == 0


@pytest.mark.parametrize("window", [1, 6, 16, 40])
def test_window_of_the_score_rule(window):
    q, k, v = rnd(23, 6, 8), rnd(23, 2, 8, seed=1), rnd(23, 2, 5, seed=2)
    got = attention_reference(q[None], k[None], v[None], True, 0.9, rule=ScoreRule(window=window))[0]
    assert torch.allclose(got, O.attend(q, k, v, 0.9, window), atol=1e-5)


@pytest.mark.parametrize("i,j,sees", [(15, 0, True), (16, 0, False), (47, 32, True), (47, 31, False), (31, 16, True), (32, 16, False), (9, 9, True), (9, 10, False)])
def test_window_edges_with_a_key_that_stands_out(i, j, sees):
    q, k, v = C.standout_case(i, j, 48, 2, 1, 16, 4)
    rule = ScoreRule(window=16)
    o = attention_reference(q[None], k[None], v[None], True, 1.0, rule=rule)[0]
    assert torch.allclose(o[i, 0], v[j, 0], atol=1e-3) == sees == (0 <= i - j < 16)
    kept, first = rule.key_ranges(i)
    part = attention_reference(q[None, i:i + 1], k[None, first:i + 1], v[None, first:i + 1], True, 1.0, rule=rule)[0]
    assert kept == 0 and torch.allclose(part[0], o[i], atol=1e-5)


def latent_case(T, H, dn, dr, dv, R, seed=0):
    """Per-head keys and values of T tokens out of cached vectors: (q, slots [T, R + dr], stacked products, keys, values)."""
    q, slots, w = rnd(T, H, dn + dr, seed=seed), rnd(T, R + dr, seed=seed + 1), rnd(H * (dn + dv), R, seed=seed + 2) * R ** -0.5
    c = slots[:, :R]
    k = torch.cat([(c @ w[:H * dn].T).view(T, H, dn), slots[:, None, R:].expand(T, H, dr)], -1)
    return q, slots, w, k, (c @ w[H * dn:].T).view(T, H, dv)


@pytest.mark.parametrize("T,H,dn,dr,dv,R", [(19, 3, 8, 4, 6, 10), (33, 1, 5, 2, 3, 4), (17, 4, 16, 8, 16, 8)])
def test_cached_vectors_give_the_attention_of_formed_keys(T, H, dn, dr, dv, R):
    q, slots, w, k, v = latent_case(T, H, dn, dr, dv, R)
    gate = rnd(T, H * dv, seed=9)
    want = O.attend(q, k, v, 0.7).reshape(T, -1) * O.sigmoid(gate)
    out = torch.empty(1, T, H, dv)
    prompt_attention_split(q[None], k[None, ..., :dn], v[None], slots[:, R:], 0.7, out, gate)
    assert torch.allclose(out.view(T, -1), want, atol=1e-5)
    rot = dict(dims=dr, base=100.0)
    pos = torch.arange(T)
    turned = q.clone()                                               # queries whose rotation gives q
    f, _ = O.frequencies(rot)
    turned[..., dn:] = O.rotate(q[..., dn:], -pos, rot)
    qa = head_product(turned.reshape(T, -1), dn + dr, w[:H * dn], H, R, dn, transposed=True, tail=dr, table=table_of(rot, pos))
    pages = torch.full((8, 8, 1, R + dr), 1e4)
    table = torch.tensor([[6, 1, 3, 5, 0]], dtype=torch.int32)
    for t in range(T):
        pages[table[0, t // 8], t % 8, 0] = slots[t]
    c = latent_decode(qa, pages, R, table.expand(T, -1), torch.arange(1, T + 1, dtype=torch.int32), 0.7)
    o = torch.empty(T, H * dv)
    head_product(c, R, w[H * dn:], H, dv, R, transposed=False, gate=gate, out=o)
    assert torch.allclose(o, want, atol=1e-4)


def test_latent_prep():
    T, qr, R, dr = 5, 12, 10, 6
    rot = dict(dims=4, base=50.0)                                    # the last two numbers of the rotated part stay
    p, gq, gk = rnd(T, 40), rnd(qr, seed=1), rnd(R, seed=2)
    before, pos, slots = p.clone(), torch.tensor([4, 0, 9, 2, 30]), torch.tensor([3, -1, 0, 7, 5])
    cache = torch.zeros(2, 4, 1, R + dr)
    latent_prep_(p, 2, qr, 20, R, dr, q_gamma=gq, kv_gamma=gk, eps=1e-2, table=table_of(rot, pos), cache=cache, slots=slots)
    want = before.clone()
    want[:, 2:14] = O.rms_norm(before[:, 2:14], gq, 1e-2)
    want[:, 20:30] = O.rms_norm(before[:, 20:30], gk, 1e-2)
    want[:, 30:36] = O.rotate(before[:, None, 30:36], pos, rot)[:, 0]
    assert torch.allclose(p, want, atol=1e-5)
    keep = slots >= 0
    assert torch.allclose(cache.view(8, -1)[slots[keep]], want[keep, 20:36], atol=1e-5) and float(cache.view(8, -1)[[1, 2, 4, 6]].abs().max()) == 0


def test_norms_around_a_sublayer():
    x, y, w, nxt = rnd(5, 16), rnd(5, 16, seed=1), rnd(16, seed=2) * 0.3, rnd(16, seed=3) * 0.3
    want = x + O.centred_norm(y, w, 1e-2)
    h = torch.empty(5, 16)
    x1 = x.clone()
    residual_norm(y, 1 + w, None, 1e-2, True, x=x1, h=h, next_gamma=1 + nxt)
    assert torch.allclose(x1, want, atol=1e-5) and torch.allclose(h, O.centred_norm(want, nxt, 1e-2), atol=1e-5)
    pair, x2 = torch.zeros(5, 32), x.clone()
    residual_norm(y, 1 + w, None, 1e-2, True, x=x2, h=pair[:, :16])            # a copy beside something else
    assert torch.equal(pair[:, :16], x2) and float(pair[:, 16:].abs().max()) == 0
    rows, slots, ws = rnd(20, 16, seed=4), torch.tensor([3, 7, 0, 19, 5, 5, 2, 1, 9, 8], dtype=torch.int32), torch.rand(5, 2)
    mixed = (rows[slots.long()].view(5, 2, 16) * ws[..., None]).sum(1)
    x3 = x.clone()
    residual_norm(rows, 1 + w, None, 1e-2, True, x=x3, h=h, next_gamma=1 + nxt, routed=(slots, ws))
    want = x + O.centred_norm(mixed, w, 1e-2)
    assert torch.allclose(x3, want, atol=1e-5) and torch.allclose(h, O.centred_norm(want, nxt, 1e-2), atol=1e-5)


ROUTERS = [(8, 2, 4, 2, 2), (12, 3, 3, 1, 2), (6, 1, 6, 1, 2), (9, 4, 3, 2, 1), (10, 10, 1, 1, 2), (1, 1, 1, 1, 2), (64, 6, 8, 4, 2)]


@pytest.mark.parametrize("E,k,groups,keep,best", ROUTERS)
def test_sigmoid_router(E, k, groups, keep, best):
    z, corr = 2 * rnd(40, E), rnd(E, seed=1) - 0.5
    idx, w = route_sigmoid(z, k, groups, keep, corr, best)
    for t in range(40 if best == 2 else 0):
        want_i, want_w = O.choose(z[t], corr, k, groups, keep)
        assert idx[t].tolist() == want_i and torch.allclose(w[t], want_w, atol=1e-6)
    i2, w2 = route_sigmoid(z, k, groups, keep, corr, best, renorm=True)
    assert torch.equal(i2, idx) and torch.allclose(w2.sum(-1), torch.ones(40), atol=1e-5)


def test_router_with_negative_choice_scores():
    """The experts of dropped groups are out even where all that is left is negative; the weights know nothing of the correction."""
    z = torch.zeros(1, 6)
    corr = torch.tensor([-3.0, -4.0, -0.1, -9.0, -2.0, -2.5])
    idx, w = route_sigmoid(z, 2, 3, 1, corr, 2)                               # sums -6, -8.1, -3.5
    assert idx.tolist() == [[4, 5]] and w.tolist() == [[0.5, 0.5]]
    assert route_sigmoid(z, 2, 3, 1, corr, 1)[0].tolist() == [[2, 3]]         # by the largest score of a group alone
    assert route_sigmoid(z, 2, 1, 1, corr, 2)[0].tolist() == [[2, 4]]


def test_clamped_gate_and_squared_relu():
    gu = 4 * rnd(7, 24)
    g, u = gu[:, :12], gu[:, 12:]
    eye = torch.eye(12)
    w = {"gate": eye, "up": eye, "down": eye}

    def want(lim):
        gg, uu = torch.clamp(g, max=lim), torch.clamp(u, -lim, lim)
        return gg * O.sigmoid(1.702 * gg) * (uu + 1)
    for lim in (0.5, 1.0, 7.0):
        assert torch.allclose(swiglu_rows(gu, act="clamped", limit=lim), want(lim), atol=1e-5)
    x = g
    assert torch.allclose(O.clamped_expert(x, w, "", 1.0), swiglu_rows(torch.cat([x, x], 1), act="clamped", limit=1.0), atol=1e-5)
    assert float(swiglu_rows(torch.tensor([[-30.0, 5.0]]), act="clamped", limit=2.0)[0, 0]) == pytest.approx(0.0, abs=1e-6)   # no lower bound on the gate
    a, b = rnd(5, 8), rnd(6, 8, seed=1)
    assert torch.allclose(gemm(a, b, act="relu2"), torch.relu(a @ b.T) ** 2, atol=1e-5) and float(act_reference("relu2", torch.tensor(-3.0))) == 0
    with pytest.raises(ValueError):
        linear(a.requires_grad_(), b, act="relu2")


def test_embedding_copy_beside_the_stream():
    t, pair = rnd(9, 8).bfloat16(), torch.zeros(2, 16, dtype=torch.bfloat16)
    x, h = embedding_residual(torch.tensor([3, 8]), t, 2.5, h=pair[:, 8:])
    assert torch.equal(x, t[[3, 8]].float() * 2.5) and torch.equal(pair[:, 8:], x.bfloat16()) and float(pair[:, :8].abs().max()) == 0


# ---- cache ----------------------------------------------------------------------------------------------------------
def test_joint_cache_layers_hold_one_array():
    c = PagedCache(4, 8, dtype=F32, layers=[CacheLayer(1, 12, 8, joint=True), CacheLayer(2, 4, 3)])
    assert c.v[0].data_ptr() == c.k[0].data_ptr() and c.v[0].shape == (4, 8, 1, 8) and c.v[1].shape == (4, 8, 2, 3)
    assert c.memory_bytes() == 4 * 4 * 8 * (12 + 2 * 4 + 2 * 3)


def test_every_pass_has_a_cache_of_its_own():
    lc = LayeredConfig.from_json(C.CONFIGS["varied"])
    assert lc.runs == ((0, None), (1, 0), (2, None), (3, None), (1, 1), (2, None), (3, None), (4, None), (5, None))
    r = C.runner(C.CONFIGS["varied"], C.weights(C.CONFIGS["varied"]))
    assert len({t.data_ptr() for t in r.cache.k}) == 9 == r.body.depth
    assert LayeredConfig.from_json(C.CONFIGS["single"]).runs[3] == (0, 1) and LayeredConfig.from_json(C.CONFIGS["straight"]).loop is None


@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_prefill_portions_and_decoding_agree_with_the_plain_model(name):
    C.check_prefill_portions_and_decode(name, "cpu", F32, 70 if name != "wide" else 40)


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


MISTAKES = {
    "window": lambda c, w: c["layers"][0]["mixer"]["mask"].update(size=21),
    "rotated dims": lambda c, w: c["layers"][0]["mixer"]["rot"].update(dims=6),
    "base": lambda c, w: c["layers"][1]["mixer"]["rot"].update(base=9000.0),
    "yarn": lambda c, w: c["layers"][1]["mixer"]["rot"].pop("scaling"),
    "yarn factor": lambda c, w: c["layers"][3]["mixer"]["rot"]["scaling"].update(factor=5.0),
    "yarn ramp": lambda c, w: c["layers"][3]["mixer"]["rot"]["scaling"].update(slow=0.02),
    "scale": lambda c, w: c["layers"][3]["mixer"].update(scale=c["layers"][3]["mixer"]["scale"] * 1.05),
    "embedding scale": lambda c, w: c["embedding"].update(scale=2.6),
    "eps": lambda c, w: c["norm"].update(eps=1e-2),
    "loop times": lambda c, w: (c["loop"].update(times=3), w.update({"loop.step": torch.cat([w["loop.step"], w["loop.step"][:1]])})),
    "loop stop": lambda c, w: c["loop"].update(stop=3),
    "loop step": lambda c, w: w.update({"loop.step": w["loop.step"].flip(0)}),
    "loop input": lambda c, w: w.update({"loop.in": w["loop.in"].roll(64, 1)}),
    "norm in front": lambda c, w: w["l2.norm1"].zero_(),
    "norm behind": lambda c, w: w["l2.norm1b"].zero_(),
    "norm behind the feed-forward": lambda c, w: w["l0.norm2b"].zero_(),
    "final norm": lambda c, w: w["final.norm"].zero_(),
    "query bias": lambda c, w: w["l0.mix.q.b"].zero_(),
    "key bias": lambda c, w: w["l2.mix.k.b"].zero_(),
    "value bias": lambda c, w: w["l2.mix.v.b"].zero_(),
    "query latent norm": lambda c, w: w["l1.mix.dq.norm"].fill_(1),
    "latent norm": lambda c, w: w["l3.mix.dkv.norm"].fill_(1),
    "output gate": lambda c, w: w["l1.mix.g"].zero_(),
    "choice correction": lambda c, w: w["l0.mlp.correction"].zero_(),
    "groups": lambda c, w: c["layers"][0]["mlp"]["router"]["groups"].update(keep=3),
    "limit": lambda c, w: c["layers"][2]["mlp"]["expert"].update(limit=0.9),
}


def _patches(monkeypatch):
    plain_frequencies, plain_choose = O.frequencies, O.choose

    def halves(x, positions, rot):
        f, m = O.frequencies(rot)
        a = positions.double()[:, None] * torch.tensor(f, dtype=torch.float64)
        c, s = (torch.cos(a) * m).to(x.dtype)[:, None], (torch.sin(a) * m).to(x.dtype)[:, None]
        n = rot["dims"]
        u, v = x[..., :n // 2], x[..., n // 2:n]
        return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], -1)

    def corrected_weights(z, corr, *a):
        idx, w = plain_choose(z, corr, *a)
        return idx, w + corr[idx]

    def normed_weights(*a):
        idx, w = plain_choose(*a)
        return idx, w / w.sum()
    return {"pairing": ("rotate", halves), "magnitude": ("frequencies", lambda rot: (plain_frequencies(rot)[0], 1.0)),
            "weights with correction": ("choose", corrected_weights), "renormed weights": ("choose", normed_weights),
            "relu": ("relu2_ff", lambda x, w, p: torch.relu(x @ w[p + "up"].T) @ w[p + "down"].T),
            "up shift": ("clamped_expert", lambda x, w, p, lim: (torch.clamp(x @ w[p + "gate"].T, max=lim) * torch.clamp(x @ w[p + "up"].T, -lim, lim)) @ w[p + "down"].T)}


PATCHED = ["pairing", "magnitude", "weights with correction", "renormed weights", "relu", "up shift"]


@pytest.mark.parametrize("mistake", [*MISTAKES, *PATCHED])
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
        name, fn = _patches(monkeypatch)[mistake]
        monkeypatch.setattr(O, name, fn)
    with pytest.raises(AssertionError):
        C.assert_logits(got, C.reference(bad, w, toks), F32)


# ---- the engine -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("prefill_chunk", [0, 8, 2048])
def test_greedy_generation_through_the_engine(prefill_chunk):
    cfg = C.CONFIGS["varied"]
    w = C.weights(cfg, 6)
    r = C.runner(cfg, w, blocks=40)
    C.poison(r)
    eng = ServingEngine(r, max_batch_size=3, prefill_chunk=prefill_chunk)
    prompts = [C.tokens(cfg, n, 20 + n) for n in (5, 19, 33, 1)]
    ids = [eng.submit(p, 5) for p in prompts]
    eng.run_to_completion()
    wd = {k: v.double() for k, v in w.items()}
    for p, rid in zip(prompts, ids):
        assert eng.scheduler.get(rid).generated == O.greedy(cfg, wd, p, 5)
    assert r.cache.free_blocks == 40


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
    assert lc.embed_scale == 2.5 and lc.norm_eps == 1e-3 and lc.layers[3].mlp is None and "head" not in lc.tensor_shapes()
    a, m = lc.layers[0].mixer, lc.layers[0].mlp
    assert a.window == 20 and a.gate == "none" and a.bias and not a.qk_norm and not a.sink and a.chunk == 0 and a.rot.dims == 8
    assert m == MoESpec(24, 8, 2, 4, 2, score="sigmoid", correction=True, group_best=2, renorm=False, act="clamped", limit=1.5)
    assert "Bikilix" in ARCHITECTURES and ARCHITECTURES["Bikilix"].float32
    p = preset("bikilix-test")
    assert p.n_layer == 4 and len(p.runs) == 6 and p.vocab_padded == 1024 and preset("bikilix-moe", n_layer=7).runs[-1] == (6, 1)
    bads = [lambda c: c["layers"][0].update(type="delta"), lambda c: c["layers"][0]["mlp"].update(kind="swiglu"), lambda c: c["loop"].update(stop=7),
            lambda c: c["loop"].update(start=4), lambda c: c["loop"].update(times=0), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26),
            lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), lambda c: c["layers"][0]["mixer"].update(kv_heads=3),
            lambda c: c["layers"][0]["mlp"]["router"].update(top=5), lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0)]
    for bad in bads:
        c = copy.deepcopy(C.CONFIGS["varied"])
        bad(c)
        with pytest.raises(ValueError):
            LayeredConfig.from_json(c)
    with pytest.raises(ValueError):
        LayeredConfig.from_json({**C.CONFIGS["varied"], "architecture": "Dolurax", "layers": C.CONFIGS["varied"]["layers"][:1]})


def test_random_weights_and_preset_run():
    from rustral_b200.serve import ModelRunner
    cfg = preset("bikilix-test")
    out = ServingEngine(ModelRunner(cfg, device="cpu", num_blocks=16)).generate([1, 2, 3], 3)
    assert len(out) == 3 and all(0 <= t < cfg.vocab_size for t in out)


def test_loading_is_strict(tmp_path):
    cfg = C.CONFIGS["varied"]
    lc, w = LayeredConfig.from_json(cfg), C.weights(cfg)
    for gone in ("l1.mix.dkv.norm", "loop.step", "l0.mix.v.b", "l0.mlp.correction"):
        with pytest.raises(SerializationError):
            InferenceWeights.layered(lc, "cpu", None, {k: v for k, v in w.items() if k != gone})
    with pytest.raises(SerializationError):
        InferenceWeights.layered(lc, "cpu", None, {**w, "head": w["embed"]})
    with pytest.raises(ShapeMismatch):
        InferenceWeights.layered(lc, "cpu", None, {**w, "l1.mix.uk": w["l1.mix.uk"][:-1]})
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
