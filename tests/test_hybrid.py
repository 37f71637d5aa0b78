"""Hybrid decoders (Vafodra) on the CPU path: each mechanism, the step function, the cache and its state slots, the engine and the
loaders against the plain restatement in tests/hybrid_oracle.py."""
import copy
import json
import os
import subprocess
import urllib.request

import numpy as np
import pytest
import torch

import hybrid_checks as C
import hybrid_oracle as O
from rustral_b200.core.errors import InvalidArgument, SerializationError, ShapeMismatch
from rustral_b200.io import safetensors_io as st
from rustral_b200.models.config import preset
from rustral_b200.models.layered import LayeredConfig
from rustral_b200.models.registry import ARCHITECTURES
from rustral_b200.ops import (ScoreRule, Segments, attention_reference, delta_rule, embedding_residual, gated_norm, short_conv, state_space,
                              stream_update)
from rustral_b200.ops.moe import swiglu_rows
from rustral_b200.serve import PagedCache, ServingEngine
from rustral_b200.serve.kv_cache import CacheLayer
from rustral_b200.serve.model_runner import load_runner
from rustral_b200.serve.weights import InferenceWeights

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32 = torch.float32


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


# ---- mechanisms ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("window,keep,sink", [(0, 0, True), (6, 0, False), (6, 2, True), (1, 0, True), (1, 3, False), (40, 5, True), (3, 30, True)])
def test_score_rule_matches_plain_attention(window, keep, sink):
    q, k, v = rnd(23, 6, 8), rnd(23, 2, 8, seed=1), rnd(23, 2, 5, seed=2)
    want = O.attention(q, k, v, 0.9, window, keep, sink)
    got = attention_reference(q[None], k[None], v[None], True, 0.9, rule=ScoreRule(window=window, keep_first=keep, sink=sink))[0]
    assert torch.allclose(got, want, atol=1e-5)


def test_sink_takes_the_weight_of_a_score_of_zero():
    q, k, v = torch.zeros(1, 1, 1, 4), torch.zeros(1, 1, 1, 4), torch.ones(1, 1, 1, 2)
    assert float(attention_reference(q, k, v, True, 1.0, rule=ScoreRule(sink=True))[0, 0, 0, 0]) == pytest.approx(0.5)
    q, k = torch.full((1, 1, 1, 1), 200.0), torch.ones(1, 1, 1, 1)
    assert float(attention_reference(q, k, v, True, 1.0, rule=ScoreRule(sink=True))[0, 0, 0, 0]) == pytest.approx(1.0)
    assert float(attention_reference(-q, k, v, True, 1.0, rule=ScoreRule(sink=True))[0, 0, 0, 0]) == pytest.approx(0.0)


@pytest.mark.parametrize("i,j,sees", [(15, 0, True), (16, 0, True), (30, 2, True), (30, 3, False), (19, 4, True), (20, 4, False), (47, 32, True),
                                      (47, 31, False), (9, 9, True)])
def test_window_edges_with_a_key_that_stands_out(i, j, sees):
    """Windows of 16 with three kept tokens: a far key inside takes nearly all weight, one token further out it takes none."""
    q, k, v = C.standout_case(i, j, 48, 2, 1, 16, 4)
    rule = ScoreRule(window=16, keep_first=3, sink=True)
    o = attention_reference(q[None], k[None], v[None], True, 1.0, rule=rule)[0]
    assert torch.allclose(o[i, 0], v[j, 0], atol=1e-3) == sees == O.visible(i, j, 16, 3)
    kept, first = rule.key_ranges(i)
    keys = [*range(kept), *range(first, i + 1)]                          # what a portion that starts at i gathers
    part = attention_reference(q[None, i:i + 1], k[None, keys], v[None, keys], True, 1.0, rule=rule)[0]
    assert torch.allclose(part[0], o[i], atol=1e-5)


def test_key_ranges_of_a_portion():
    rule = ScoreRule(window=10, keep_first=4)
    assert rule.key_ranges(0) == (0, 0) and rule.key_ranges(13) == (0, 0) and rule.key_ranges(14) == (4, 5)
    assert ScoreRule(window=10).key_ranges(14) == (0, 5)
    assert ScoreRule(slopes=torch.ones(2), window=10, keep_first=4).key_ranges(50) == (0, 0)
    assert ScoreRule(chunk=8).key_ranges(21) == (0, 16)


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
@pytest.mark.parametrize("cuts", [[], [1, 2, 3], [2, 11], [5, 6, 12]])
def test_short_conv_carries_its_last_inputs(taps, cuts):
    x, w, b = rnd(17, 5), rnd(5, taps, seed=1), rnd(5, seed=2)
    want = O.silu(O.causal_conv(x, w, b))
    state = torch.full((3, taps - 1, 5), 9.0)
    got, lo = [], 0
    for hi in [*cuts, 17]:
        got.append(short_conv(x[lo:hi], w, b, state, Segments.of([(0, hi - lo, 1, lo)], "cpu")))
        lo = hi
    assert torch.allclose(torch.cat(got), want, atol=1e-5)
    assert bool((state[[0, 2]] == 9.0).all())
    assert torch.allclose(short_conv(x, w, None, state, Segments.of([(0, 17, 0, 0)], "cpu"), silu=False), O.causal_conv(x, w), atol=1e-5)


@pytest.mark.parametrize("H,G,P,N", [(4, 2, 6, 5), (1, 1, 8, 3), (6, 1, 4, 4), (3, 3, 5, 2)])
def test_state_space_over_unequal_segments(H, G, P, N):
    T, inner = 19, H * P
    xbc, dt = rnd(T, inner + 2 * G * N), rnd(T, H, seed=1)
    bias, a_log, D = rnd(H, seed=2), rnd(H, seed=3), rnd(H, seed=4)
    x, B, Cm = xbc[:, :inner].reshape(T, H, P), xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    kw = dict(dt_bias=bias, a_log=a_log, D=D, heads=H, groups=G, vdim=P, n=N)
    state = torch.full((4, H, N, (P + 3) // 4 * 4), 7.0)
    segs = [(0, 12, 2, 0), (12, 1, 0, 0), (13, 6, 3, 0)]
    y = state_space(xbc, dt, state=state, seg=Segments.of(segs, "cpu"), **kw)
    want = C.oracle_state_space(segs, x, B, Cm, dt, bias, a_log, D, {})
    assert torch.allclose(y.view(T, H, P), want, atol=1e-4)
    more = state_space(xbc[13:], dt[13:], state=state, seg=Segments.of([(0, 6, 2, 12)], "cpu"), **kw)       # sequence 2 goes on
    past = {0: (x[:12], B[:12], Cm[:12], dt[:12])}
    want = C.oracle_state_space([(0, 6, 2, 12)], x[13:], B[13:], Cm[13:], dt[13:], bias, a_log, D, past)
    assert torch.allclose(more.view(6, H, P), want, atol=1e-4) and bool((state[1] == 7.0).all())


def test_state_space_decays_before_it_takes_up_the_token():
    """One head, state of one row: y_1 sees its own write, y_2 the first one decayed once."""
    xbc = torch.tensor([[2.0, 1.0, 1.0], [0.0, 1.0, 1.0]])                # x, B, C
    zero = torch.zeros(1)
    y = state_space(xbc, torch.tensor([[0.3], [0.7]]), dt_bias=zero, a_log=torch.tensor([0.5]), D=torch.tensor([10.0]), heads=1, groups=1,
                    vdim=1, n=1, state=torch.zeros(1, 1, 1, 4), seg=Segments.of([(0, 2, 0, 0)], "cpu"))
    d1, d2 = np.log1p(np.exp(0.3)), np.log1p(np.exp(0.7))
    assert float(y[0]) == pytest.approx(2 * d1 + 20.0, rel=1e-5) and float(y[1]) == pytest.approx(2 * d1 * np.exp(-np.exp(0.5) * d2), rel=1e-5)


@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 6, 5), (1, 1, 8, 3), (6, 2, 4, 4), (3, 3, 5, 2)])
def test_delta_rule_over_unequal_segments(H, G, dk, dv):
    T, nk = 19, G * dk
    qkv, ab = rnd(T, 2 * nk + H * dv), rnd(T, 2 * H, seed=1)
    bias, a_log = rnd(H, seed=2), rnd(H, seed=3)
    q = O.unit(qkv[:, :nk].reshape(T, G, dk)) * dk ** -0.5
    k, v = O.unit(qkv[:, nk:2 * nk].reshape(T, G, dk)), qkv[:, 2 * nk:].reshape(T, H, dv)
    beta, decay = O.sigmoid(ab[:, H:]), torch.exp(-torch.exp(a_log) * O.softplus(ab[:, :H] + bias))
    state = torch.full((3, H, dk, (dv + 3) // 4 * 4), 7.0)
    kw = dict(dt_bias=bias, a_log=a_log, state=state, heads=H, kv_heads=G, dk=dk, dv=dv)
    want = O.gated_delta(q, k, v, beta, decay)
    for first, n in ((0, 7), (7, 1), (8, 11)):                            # one sequence in three portions
        o = delta_rule(qkv[first:first + n], ab[first:first + n, :H], ab[first:first + n, H:], seg=Segments.of([(0, n, 1, first)], "cpu"), **kw)
        assert torch.allclose(o.view(n, H, dv), want[first:first + n], atol=1e-4)
    two = delta_rule(qkv, ab[:, :H], ab[:, H:], seg=Segments.of([(0, 9, 2, 0), (9, 10, 0, 0)], "cpu"), **kw)
    assert torch.allclose(two[:9].view(9, H, dv), want[:9], atol=1e-4)
    assert torch.allclose(two[9:].view(10, H, dv), O.gated_delta(q[9:], k[9:], v[9:], beta[9:], decay[9:]), atol=1e-4)


def test_delta_rule_replaces_what_a_key_held():
    """beta near 1 and no decay: the second write at the same key replaces the first value instead of adding to it."""
    qkv = torch.tensor([[1.0, 0.0, 1.0, 0.0, 5.0], [1.0, 0.0, 1.0, 0.0, -3.0]])
    o = delta_rule(qkv, torch.full((2, 1), -40.0), torch.full((2, 1), 40.0), dt_bias=torch.zeros(1), a_log=torch.zeros(1), heads=1, kv_heads=1,
                   dk=2, dv=1, state=torch.zeros(1, 1, 2, 4), seg=Segments.of([(0, 2, 0, 0)], "cpu"))
    assert torch.allclose(o * 2 ** 0.5, torch.tensor([[5.0], [-3.0]]), atol=1e-4)


def test_gated_norms():
    y, z, w = rnd(6, 24), rnd(6, 24, seed=1), rnd(24, seed=2)
    for parts in (1, 3, 8):
        assert torch.allclose(gated_norm(y, z, w, parts, 1e-2, True), O.gated_group_norm(y, z, w, parts, 1e-2), atol=1e-5)
    want = O.rms_norm(y.view(6, 4, 6), w[:6], 1e-2) * O.silu(z).view(6, 4, 6)
    assert torch.allclose(gated_norm(y, z, w[:6], 4, 1e-2, False), want.reshape(6, 24), atol=1e-5)


def test_stream_update_and_dynamic_tanh():
    x, a, b, c = (rnd(5, 16, seed=i) for i in range(4))
    wa, wb, g, beta, alpha = rnd(16, seed=5), rnd(16, seed=6), rnd(16, seed=7), rnd(16, seed=8), torch.tensor([0.7])
    want = x + 0.3 * (0.5 * (O.rms_norm(a, wa, 1e-3) + O.rms_norm(b, wb, 1e-3)) + c)
    x1, h = x.clone(), torch.empty(5, 16)
    stream_update(x1, a=a, wa=wa, b=b, wb=wb, c=c, normed=0.5, mult=0.3, eps=1e-3, dyt=(g, beta, alpha), h=h)
    assert torch.allclose(x1, want, atol=1e-5) and torch.allclose(h, O.dynamic_tanh(want, alpha, g, beta), atol=1e-5)
    x2 = x.clone()
    assert torch.allclose(stream_update(x2, c=c, mult=0.3), x + 0.3 * c, atol=1e-6)
    x3 = x.clone()
    assert torch.allclose(stream_update(x3, dyt=(g, beta, alpha)), O.dynamic_tanh(x, alpha, g, beta), atol=1e-5) and torch.equal(x3, x)


def test_embedding_scale_and_relu_gate():
    t = rnd(9, 8).bfloat16()
    x, h = embedding_residual(torch.tensor([3, 8]), t, 2.5, want_h=False)
    assert h is None and torch.equal(x, t[[3, 8]].float() * 2.5)
    gu = rnd(4, 12)
    assert torch.allclose(swiglu_rows(gu, act="relu"), torch.relu(gu[:, :6]) * gu[:, 6:])
    out = torch.zeros(4, 10)
    swiglu_rows(gu, act="relu", out=out[:, 2:8])
    assert torch.equal(out[:, 2:8], swiglu_rows(gu, act="relu")) and float(out[:, [0, 1, 8, 9]].abs().max()) == 0
    with pytest.raises(ValueError):
        swiglu_rows(gu, act="gelu")


# ---- cache and state slots ------------------------------------------------------------------------------------------
def test_state_slots_are_held_from_allocate_to_free():
    layers = [CacheLayer(2, 4, 3, (("conv", (3, 5), None), ("state", (2, 4, 4), torch.float32))), CacheLayer(state=(("state", (1, 2, 4), F32),))]
    c = PagedCache(8, 4, dtype=torch.bfloat16, layers=layers, num_slots=2)
    assert c.k[1] is None and c.state[0]["conv"].shape == (2, 3, 5) and c.state[0]["conv"].dtype == torch.bfloat16
    assert c.allocate(10, 3) and c.allocate(11, 1)
    a, b = c.state_slot(10), c.state_slot(11)
    assert {a, b} == {0, 1} and c.free_slots == 0
    assert not c.can_allocate(12, 1) and not c.allocate(12, 1) and c.state_slot(12) == -1 and c.block_table(12) == []
    assert c.allocate(10, 9) and c.state_slot(10) == a                   # growing keeps the slot
    assert not c.allocate(10, 1000) and c.state_slot(10) == a
    c.free(11)
    assert c.allocate(12, 2) and c.state_slot(12) == b
    c.free(10)
    c.free(12)
    assert c.free_slots == 2 and c.free_blocks == 8 and c.memory_bytes() > 0
    with pytest.raises(InvalidArgument):
        PagedCache(8, 4, layers=layers, num_slots=0)
    plain = PagedCache(8, 4, layers=[CacheLayer(1, 4, 4)], num_slots=1)
    assert plain.num_slots == 0 and plain.allocate(1, 1) and plain.allocate(2, 1) and plain.state_slot(1) == -1


def test_segments_split_and_tiles():
    s = Segments.of([(0, 40, 3, 0), (40, 1, 1, 7), (41, 17, 0, 2), (58, 1, 2, 0)], "cpu")
    many, one = s.split()
    assert many.rows == [(0, 40, 3, 0), (41, 17, 0, 2)] and one.rows == [(40, 1, 1, 7), (58, 1, 2, 0)]
    assert many.table.tolist() == [list(r) for r in many.rows] and one.single and not s.single
    assert s.tiles(16).tolist() == [[0, 0], [0, 16], [0, 32], [1, 0], [2, 0], [2, 16], [3, 0]]
    assert one.tiles(16).tolist() == [[0, 0], [1, 0]] and one.split() == (None, one)


@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_prefill_portions_and_decoding_agree_with_the_plain_model(name):
    C.check_prefill_portions_and_decode(name, "cpu", F32, 70 if name != "wide" else 40)


@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_mixed_batches_with_reused_pages_and_slots(name):
    C.check_mixed_batch_with_reused_pages_and_slots(name, "cpu", F32)


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


def test_layers_that_share_tensors_have_a_cache_and_state_of_their_own():
    cfg = C.CONFIGS["varied"]
    lc = LayeredConfig.from_json(cfg)
    assert [lc.owner(i) for i in range(8)] == [0, 1, 2, 0, 1, 6, 6, 0]
    assert not any(n.startswith(("l3.", "l4.", "l5.", "l7.")) for n in lc.tensor_shapes())
    r = C.runner(cfg, C.weights(cfg))
    held = [t.data_ptr() for d in r.cache.state for t in d.values() if t.numel()] + [t.data_ptr() for t in r.cache.k if t is not None]
    assert len(set(held)) == len(held) == 16 + 4
    for bad in ({"weights_of": 1}, {"weights_of": 99}):
        c = copy.deepcopy(cfg)
        c["layers"][3].update(bad)
        with pytest.raises(ValueError):
            LayeredConfig.from_json(c)


@pytest.mark.parametrize("mistake", ["window", "keep", "sink", "head gate", "eps", "decay", "D", "norm parts", "conv bias", "beta", "unit", "alpha",
                                     "scale", "mult", "filter", "gate order"])
def test_the_comparison_notices_a_mistake(mistake, monkeypatch):
    """The plain model with one thing changed must not agree: the checks above would see such a fault."""
    cfg = C.CONFIGS["varied"]
    w = {k: v.clone() for k, v in C.weights(cfg).items()}
    toks = C.tokens(cfg, 60)
    got = C.feed(C.runner(cfg, w), 0, toks, [])
    bad = copy.deepcopy(cfg)
    if mistake == "window":
        bad["layers"][2]["mixer"]["left"]["mask"]["size"] += 1
    elif mistake == "keep":
        bad["layers"][2]["mixer"]["left"]["mask"]["keep_first"] -= 1
    elif mistake == "sink":
        plain = O.attention
        monkeypatch.setattr(O, "attention", lambda *a: plain(*a, sink=False))
    elif mistake == "head gate":
        w["l0.mix.left.g"].zero_()
    elif mistake == "eps":
        bad["norm"]["eps"] = 1e-2
    elif mistake == "decay":
        w["l1.mix.A_log"] += 0.2
    elif mistake == "D":
        w["l2.mix.right.D"].zero_()
    elif mistake == "norm parts":
        bad["layers"][0]["mixer"]["right"]["norm_groups"] = 1
    elif mistake == "conv bias":
        w["l0.mix.right.conv.b"].zero_()
    elif mistake == "beta":
        w["l1.mix.b"].zero_()
    elif mistake == "unit":
        monkeypatch.setattr(O, "unit", lambda t: t / torch.sqrt((t * t).mean(-1, keepdim=True) + 1e-6))
    elif mistake == "alpha":
        w["l2.norm1.alpha"] += 0.1
    elif mistake == "scale":
        bad["embedding"]["scale"] *= 1.05
    elif mistake == "mult":
        bad["residual_mult"] *= 1.05
    elif mistake == "filter":
        w["l1.mix.k.conv"] = w["l1.mix.k.conv"].flip(1)
    else:
        monkeypatch.setattr(O, "gated_group_norm", lambda y, z, wt, n, eps: O.silu(z) * O.gated_group_norm_plain(y, wt, n, eps))
        monkeypatch.setattr(O, "gated_group_norm_plain", lambda y, wt, n, eps: (
            (u := y.view(y.shape[0], n, -1)) / torch.sqrt((u * u).mean(-1, keepdim=True) + eps)).reshape(y.shape) * wt, raising=False)
    with pytest.raises(AssertionError):
        C.assert_logits(got, C.reference(bad, w, toks), F32)


# ---- the engine -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("prefill_chunk", [0, 8, 2048])
def test_greedy_generation_through_the_engine(prefill_chunk):
    """Four requests on two state slots: admission waits for a slot, and a slot's next owner starts from zero."""
    cfg = C.CONFIGS["varied"]
    w = C.weights(cfg, 6)
    r = C.runner(cfg, w, blocks=40, slots=2)
    C.poison(r)
    eng = ServingEngine(r, max_batch_size=4, prefill_chunk=prefill_chunk)
    prompts = [C.tokens(cfg, n, 20 + n) for n in (5, 19, 33, 1)]
    ids = [eng.submit(p, 5) for p in prompts]
    eng.step()
    assert len(eng.scheduler.running) == 2 and len(eng.scheduler.pending) == 2
    eng.run_to_completion()
    wd = {k: v.double() for k, v in w.items()}
    for p, rid in zip(prompts, ids):
        assert eng.scheduler.get(rid).generated == O.greedy(cfg, wd, p, 5)
    assert r.cache.free_blocks == 40 and r.cache.free_slots == 2


def test_engine_recomputes_a_request_that_was_paused_for_memory():
    cfg = C.CONFIGS["single"]
    w = C.weights(cfg, 7)
    eng = ServingEngine(C.runner(cfg, w, blocks=6, block_size=4, slots=4), max_batch_size=4, prefill_chunk=4)
    prompts = [C.tokens(cfg, n, 40 + n) for n in (7, 6, 5)]
    ids = [eng.submit(p, 9) for p in prompts]
    eng.run_to_completion()
    wd = {k: v.double() for k, v in w.items()}
    assert eng.scheduler.stats.preempted > 0
    for p, rid in zip(prompts, ids):
        assert eng.scheduler.get(rid).generated == O.greedy(cfg, wd, p, 9)


def test_abort_gives_the_slot_back():
    cfg = C.CONFIGS["single"]
    r = C.runner(cfg, C.weights(cfg), slots=1)
    eng = ServingEngine(r, prefill_chunk=4)
    a, b = eng.submit(C.tokens(cfg, 20), 4), eng.submit(C.tokens(cfg, 3), 2)
    eng.step()
    assert r.cache.free_slots == 0 and eng.abort(a)
    eng.run_to_completion()
    assert len(eng.scheduler.get(b).generated) == 2 and r.cache.free_slots == 1


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
    assert lc.embed_scale == 3.5 and lc.residual_mult == 0.7 and lc.norm_eps == 1e-3 and lc.layers[2].mlp is None
    a = lc.layers[0].mixer.left
    assert a.sink and a.gate == "head" and a.window == 20 and a.keep_first == 3 and not a.qk_norm and not a.distance_bias and a.chunk == 0
    assert "Vafodra" in ARCHITECTURES and ARCHITECTURES["Vafodra"].float32
    p = preset("vafodra-test")
    assert p.n_layer == 4 and p.owner(2) == 0 and p.vocab_padded == 1024 and preset("vafodra-8b", n_layer=3).n_layer == 3
    bads = [lambda c: c["layers"][0].update(type="recurrent"), lambda c: c["layers"][0]["mlp"].update(kind="moe"),
            lambda c: c["layers"][0]["mixer"]["right"].update(groups=4), lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=5),
            lambda c: c["layers"][1]["mixer"].update(kv_heads=4), lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3)]
    for bad in bads:
        c = copy.deepcopy(C.CONFIGS["varied"])
        bad(c)
        with pytest.raises(ValueError):
            LayeredConfig.from_json(c)


def test_random_weights_and_preset_run():
    from rustral_b200.serve import ModelRunner
    cfg = preset("vafodra-test")
    r = ModelRunner(cfg, device="cpu", num_blocks=16, num_slots=2)
    out = ServingEngine(r).generate([1, 2, 3], 3)
    assert len(out) == 3 and all(0 <= t < cfg.vocab_size for t in out)


def test_loading_is_strict(tmp_path):
    cfg = C.CONFIGS["varied"]
    lc, w = LayeredConfig.from_json(cfg), C.weights(cfg)
    with pytest.raises(SerializationError):
        InferenceWeights.layered(lc, "cpu", None, {k: v for k, v in w.items() if k != "l1.mix.v.conv"})
    with pytest.raises(SerializationError):
        InferenceWeights.layered(lc, "cpu", None, {**w, "l3.mix.left.q": w["l0.mix.left.q"]})       # a sharer has no tensors
    with pytest.raises(ShapeMismatch):
        InferenceWeights.layered(lc, "cpu", None, {**w, "l0.mix.right.in": w["l0.mix.right.in"][:-1]})
    save_model(tmp_path, cfg, w)
    r = load_runner(str(tmp_path), device="cpu", num_slots=1)
    toks = C.tokens(cfg, 30)
    C.assert_logits(C.feed(r, 0, toks, [11]), C.reference(cfg, w, toks), F32)


def test_trace_replay_program(tmp_path):
    cfg = C.CONFIGS["varied"]
    w = C.weights(cfg, 11)
    save_model(tmp_path, cfg, w)
    reqs = {f"r{i}": C.tokens(cfg, n, i) for i, n in enumerate((40, 21, 9, 30, 12, 5))}
    want = {k: C.reference(cfg, w, t) for k, t in reqs.items()}
    steps, expect, at = [], {}, {k: 0 for k in reqs}

    def step(entries, end=()):
        rows, ents = [], []
        for rid, n, places in entries:
            lo = at[rid]
            ents.append({"id": rid, "tokens": reqs[rid][lo:lo + n], "want": places})
            rows += [want[rid][lo + p] for p in places]
            at[rid] += n
        if rows:
            expect[len(steps)] = torch.stack(rows)
        steps.append({"step": len(steps), "entries": ents, "end": list(end)})
    step([("r0", 17, [0, 16]), ("r1", 1, [])])
    step([("r1", 19, [18, 3]), ("r0", 1, [0]), ("r2", 2, [1]), ("r3", 7, [])])
    step([("r0", 1, [0]), ("r1", 1, [0]), ("r2", 7, [6, 0])], ["r1", "r2"])
    step([("r4", 12, [11]), ("r5", 2, [0, 1]), ("r0", 21, [20]), ("r3", 2, [])], ["r4", "r0"])
    step([("r3", 21, [0, 20]), ("r5", 3, [2])], ["r3", "r5"])
    out = tmp_path / "out"
    out.mkdir()
    res = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out),
                          "--max-tokens", "160", "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                         capture_output=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [x for x in res.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    assert sorted(os.listdir(out)) == sorted(f"{i}.f32" for i in expect)
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
