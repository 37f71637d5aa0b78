"""Layered decoders (Dolurax) on the CPU path: each mechanism, the step function, the cache, the engine and the loaders
against the plain restatement in tests/layered_oracle.py."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import layered_checks as C
import layered_oracle as O
from rustral_b200.core.errors import SerializationError, ShapeMismatch
from rustral_b200.io import safetensors_io as st
from rustral_b200.models.config import preset
from rustral_b200.models.layered import LayeredConfig
from rustral_b200.models.registry import ARCHITECTURES, load_config
from rustral_b200.ops import ScoreRule, attention_reference, distance_slopes, head_prep_, residual_norm
from rustral_b200.ops import moe as moe_ops
from rustral_b200.serve import ServingEngine
from rustral_b200.serve.model_runner import load_runner
from rustral_b200.serve.trace_run import TraceReplay
from rustral_b200.serve.weights import InferenceWeights

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32 = torch.float32


# ---- mechanisms ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("cap,chunk", [(0.0, 0), (5.0, 0), (0.0, 6), (5.0, 6), (5.0, 1), (5.0, 40)])
def test_score_rule_matches_plain_attention(cap, chunk):
    g = torch.Generator().manual_seed(0)
    q, k, v = torch.randn(23, 6, 8, generator=g), torch.randn(23, 2, 8, generator=g), torch.randn(23, 2, 5, generator=g)
    want = O.attention(q, k, v, 0.9, cap, chunk)
    got = attention_reference(q[None], k[None], v[None], True, 0.9, rule=ScoreRule(cap, distance_slopes(6), chunk))[0]
    assert torch.allclose(got, want, atol=1e-5)


def test_distance_slopes_are_a_geometric_sequence():
    assert distance_slopes(4).tolist() == [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8]
    assert distance_slopes(1).tolist() == [2.0 ** -8]
    assert torch.allclose(distance_slopes(6), O.head_slopes(6).float())


def test_distance_bias_is_taken_off_after_the_cap():
    """With the bias inside the cap, or counted from the sequence's start under a cap, the weights would differ."""
    q = torch.full((1, 4, 1, 2), 3.0)
    k = torch.tensor([4.0, 3.0, 2.0, 1.0]).view(1, 4, 1, 1).expand(1, 4, 1, 2)
    v = torch.eye(4).view(1, 4, 1, 4)
    rule = ScoreRule(2.0, torch.tensor([0.7]))
    p = attention_reference(q, k, v, True, 0.5, rule=rule)[0, 3, 0]
    s = torch.tensor([2.0 * np.tanh(6.0 * x * 0.5 / 2.0) - 0.7 * d for x, d in ((4, 3), (3, 2), (2, 1), (1, 0))])
    assert torch.allclose(p, torch.softmax(s.float(), 0), atol=1e-6)


@pytest.mark.parametrize("i,j,sees", [(15, 0, True), (16, 15, False), (31, 16, True), (32, 31, False), (47, 33, True), (16, 16, True)])
def test_chunk_edges_with_a_key_that_stands_out(i, j, sees):
    """Chunks of 16: a far key inside the chunk takes nearly all weight, one token across the edge it takes none."""
    q, k, v = C.standout_case(i, j, 48, 2, 1, 16, 4)
    o = attention_reference(q[None], k[None], v[None], True, 1.0, rule=ScoreRule(0.0, None, 16))[0]
    assert torch.allclose(o[i, 0], v[j, 0], atol=1e-3) == sees
    assert torch.allclose(o, O_no_bias(q, k, v, 16), atol=1e-5)


def O_no_bias(q, k, v, chunk):
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[2])
    for i in range(T):
        js = [j for j in range(T) if O.visible(i, j, chunk)]
        for h in range(H):
            s = torch.tensor([float(q[i, h] @ k[j, 0]) for j in js])
            out[i, h] = torch.softmax(s, 0) @ v[js, 0]
    return out


@pytest.mark.parametrize("E,k,groups,keep", [(16, 2, 2, 1), (12, 3, 3, 2), (8, 8, 1, 1), (8, 1, 8, 1), (6, 2, 6, 2), (5, 2, 1, 1)])
def test_router_chooses_inside_the_best_groups(E, k, groups, keep):
    logits = torch.randn(40, E, generator=torch.Generator().manual_seed(E))
    idx, w = moe_ops.route_groups(logits, k, groups, keep)
    s = torch.softmax(logits, -1)
    for t in range(40):
        want = O.choose_experts(s[t], k, {"count": groups, "keep": keep})
        assert idx[t].tolist() == want
        tot = sum(s[t, i] for i in want) + 1e-20
        assert torch.allclose(w[t], torch.stack([s[t, i] / tot for i in want]), atol=1e-6)


def test_router_group_limit_excludes_a_large_score():
    z = torch.tensor([[5.0, -9.0, 4.0, 3.9]])               # best expert 0; the second best, 2, is in the other group
    assert moe_ops.route_groups(z, 2, 2, 1)[0].tolist() == [[0, 1]]
    assert moe_ops.route_groups(z, 2, 2, 2)[0].tolist() == [[0, 2]]


def test_residual_norm_adds_the_norm_of_the_output():
    g = torch.Generator().manual_seed(1)
    y, x, w, b = torch.randn(7, 24, generator=g), torch.randn(7, 24, generator=g), torch.randn(24, generator=g), torch.randn(24, generator=g)
    x0, h = x.clone(), torch.empty(7, 24)
    residual_norm(y, w, b, 1e-3, x=x, h=h)
    assert torch.allclose(x, x0 + O.layer_norm(y, w, b, 1e-3), atol=1e-5) and torch.equal(x, h)
    slot, wt = torch.randperm(14, generator=g).to(torch.int32), torch.rand(7, 2, generator=g)
    rows, add, x = torch.randn(14, 24, generator=g), torch.randn(7, 24, generator=g), x0.clone()
    residual_norm(rows, w, None, 1e-3, True, x=x, routed=(slot, wt), add=add)
    src = add + wt[:, :1] * rows[slot[0::2].long()] + wt[:, 1:] * rows[slot[1::2].long()]
    assert torch.allclose(x, x0 + O.rms_norm(src, w, 1e-3), atol=1e-5)


def test_head_prep_norms_mixes_and_stores():
    g = torch.Generator().manual_seed(2)
    H, G, dk, dv, T = 4, 2, 6, 3, 5
    p = torch.randn(T, H * dk + G * (dk + dv) + 4, generator=g)
    p0, first = p.clone(), torch.randn(T, G * dv, generator=g)
    kc, vc = torch.zeros(3, 4, G, dk), torch.zeros(3, 4, G, dv)
    slots = torch.tensor([3, 7, -1, 0, 11])
    qg, kg, lam = torch.randn(dk, generator=g), torch.randn(dk, generator=g), torch.tensor([0.3])
    head_prep_(p, H, G, dk, dv, q_gamma=qg, k_gamma=kg, eps=1e-4, v_first=first, mix=lam, k_cache=kc, v_cache=vc, slots=slots)
    q = O.rms_norm(p0[:, :H * dk].view(T, H, dk), qg, 1e-4)
    k = O.rms_norm(p0[:, H * dk:(H + G) * dk].view(T, G, dk), kg, 1e-4)
    v = O.mix_values(p0[:, (H + G) * dk:(H + G) * dk + G * dv], first, 0.3).view(T, G, dv)
    assert torch.allclose(p[:, :H * dk].view(T, H, dk), q, atol=1e-5) and torch.equal(p[:, -4:], p0[:, -4:])
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.allclose(kc.view(12, G, dk)[s], k[t], atol=1e-5) and torch.allclose(vc.view(12, G, dv)[s], v[t], atol=1e-5)
    assert float(kc.view(12, -1)[[1, 2, 4, 5, 6, 8, 9, 10]].abs().max()) == 0


# ---- the step function and the cache ------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_prefill_portions_and_decoding_agree_with_the_plain_model(name):
    C.check_prefill_portions_and_decode(name, "cpu", F32)


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
    toks = C.tokens(cfg, 60, 3)
    r = C.runner(cfg, w, blocks=128, block_size=block_size)
    C.assert_logits(C.feed(r, 0, toks, [5, 7, 33, 34, 35]), C.reference(cfg, w, toks), F32, block_size)


@pytest.mark.parametrize("mistake", ["chunk", "slope", "gate", "cap", "mix", "groups", "eps"])
def test_the_comparison_notices_a_wrong_constant(mistake, monkeypatch):
    """The plain model with one constant changed must not agree: the checks above would see such a fault."""
    cfg = C.CONFIGS["varied"]
    w = {k: v.clone() for k, v in C.weights(cfg).items()}
    toks = C.tokens(cfg, 60)
    got = C.feed(C.runner(cfg, w), 0, toks, [])
    bad = json.loads(json.dumps(cfg))
    if mistake == "chunk":
        bad["layers"][1]["mixer"]["mask"]["size"] += 1
    elif mistake == "slope":
        monkeypatch.setattr(O, "head_slopes", lambda H, dtype: torch.tensor([2.0 ** (-8.0 * h / H) for h in range(H)], dtype=dtype))
    elif mistake == "gate":
        w["l0.mix.g"].zero_()
    elif mistake == "cap":
        bad["layers"][0]["mixer"]["softcap"] = 30.0
    elif mistake == "mix":
        w["l2.mix.vmix"].zero_()
    elif mistake == "groups":
        bad["layers"][0]["mlp"]["router"]["groups"]["keep"] = 1
    else:
        bad["norm"]["eps"] = 1e-2
    with pytest.raises(AssertionError):
        C.assert_logits(got, C.reference(bad, w, toks), F32)


# ---- the engine -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("prefill_chunk", [0, 8, 2048])
def test_greedy_generation_through_the_engine(prefill_chunk):
    cfg = C.CONFIGS["varied"]
    w = C.weights(cfg, 6)
    eng = ServingEngine(C.runner(cfg, w, blocks=40), max_batch_size=3, prefill_chunk=prefill_chunk)
    prompts = [C.tokens(cfg, n, 20 + n) for n in (5, 19, 33, 1)]
    ids = [eng.submit(p, 6) for p in prompts]
    eng.run_to_completion()
    wd = {k: v.double() for k, v in w.items()}
    for p, rid in zip(prompts, ids):
        assert eng.scheduler.get(rid).generated == O.greedy(cfg, wd, p, 6)
    assert eng.runner.cache.free_blocks == 40


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


def test_config_round_trip_and_registry(tmp_path):
    for cfg in C.CONFIGS.values():
        lc = LayeredConfig.from_json(cfg)
        assert LayeredConfig.from_json(lc.to_json()) == lc
    lc = LayeredConfig.from_json(C.CONFIGS["varied"])
    assert lc.first_mix == 1 and lc.layers[2].mlp is None and lc.layers[3].mixer.chunk == 0 and "Dolurax" in ARCHITECTURES
    assert lc.num_parameters() == sum(int(np.prod(s)) for n, s in lc.tensor_shapes().items() if not n.endswith("vmix"))
    p = preset("dolurax-test")
    assert p.n_layer == 3 and p.vocab_padded == 1024
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "llama", "vocab_size": 64, "n_head": 4, "d_model": 64, "n_layer": 1}))
    assert load_config(str(tmp_path)).arch == "llama"
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "unheard-of"}))
    with pytest.raises(ValueError):
        load_config(str(tmp_path))
    for bad in ({"heads": 3, "kv_heads": 2}, {"mask": {"size": -1}}):
        c = json.loads(json.dumps(C.CONFIGS["single"]))
        c["layers"][0]["mixer"].update(bad)
        with pytest.raises(ValueError):
            LayeredConfig.from_json(c)


def test_loading_is_strict(tmp_path):
    cfg = C.CONFIGS["varied"]
    lc, w = LayeredConfig.from_json(cfg), C.weights(cfg)
    InferenceWeights.layered(lc, "cpu", None, {**w, "l0.mix.vmix": torch.ones(())})      # unused, may be there
    with pytest.raises(SerializationError):
        InferenceWeights.layered(lc, "cpu", None, {k: v for k, v in w.items() if k != "l1.mix.g"})
    with pytest.raises(SerializationError):
        InferenceWeights.layered(lc, "cpu", None, {**w, "l0.mix.bias": torch.ones(3)})
    with pytest.raises(ShapeMismatch):
        InferenceWeights.layered(lc, "cpu", None, {**w, "head": w["head"][:-1]})
    save_model(tmp_path, cfg, w)
    r = load_runner(str(tmp_path), device="cpu")
    toks = C.tokens(cfg, 30)
    C.assert_logits(C.feed(r, 0, toks, [11]), C.reference(cfg, w, toks), F32)


def test_trace_replay_program(tmp_path):
    cfg = C.CONFIGS["varied"]
    w = C.weights(cfg, 11)
    save_model(tmp_path, cfg, w)
    a, b = C.tokens(cfg, 40, 1), C.tokens(cfg, 21, 2)
    wa, wb = C.reference(cfg, w, a), C.reference(cfg, w, b)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:17], "want": [0, 16]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:1], "want": []}, {"id": "a", "tokens": a[17:18], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[1:20], "want": [18, 3]}, {"id": "a", "tokens": a[18:19], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[19:20], "want": [0]}, {"id": "b", "tokens": b[20:], "want": [0]}], "end": ["b"]},
             {"step": 4, "entries": [{"id": "a", "tokens": a[20:], "want": [19]}], "end": ["a"]},
             {"step": 5, "entries": [{"id": "b", "tokens": b, "want": [20]}], "end": ["b"]}]
    want = {0: wa[[0, 16]], 2: torch.stack([wb[19], wb[4], wa[18]]), 3: torch.stack([wa[19], wb[20]]), 4: wa[[39]], 5: wb[[20]]}
    out = tmp_path / "out"
    out.mkdir()
    res = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out),
                          "--max-tokens", "128", "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                         capture_output=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [x for x in res.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(6)]
    assert sorted(os.listdir(out)) == [f"{i}.f32" for i in want]
    for i, x in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"])
        assert got.shape == x.shape
        C.assert_logits(got, x, F32, i)


def test_trace_replay_refuses_what_does_not_fit():
    cfg = C.CONFIGS["single"]
    rep = TraceReplay(C.runner(cfg, C.weights(cfg), blocks=2))
    rep.step([{"id": "x", "tokens": [1] * 32, "want": []}], [])
    with pytest.raises(RuntimeError):
        rep.step([{"id": "x", "tokens": [1], "want": []}], [])


def test_trace_replay_refuses_32_bit_for_families_that_lack_it(tmp_path):
    from rustral_b200.serve.trace_run import main
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "llama", "vocab_size": 64, "n_head": 4, "d_model": 64, "n_layer": 1}))
    assert main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"]) == 3


def test_kernel_files_of_every_architecture_exist_and_cover_what_they_include():
    from rustral_b200 import _build
    for a in ARCHITECTURES.values():
        for stem in a.kernels:
            assert (_build.CSRC / "kernels" / f"{stem}.cu").exists(), (a.name, stem)
    heads = list((_build.CSRC / "kernels").glob("*.h")) + list((_build.CSRC / "kernels").glob("*.cuh"))
    names = {h.name for h in _build._included(_build.CSRC / "kernels" / "moe.cu", heads)}
    assert names == {"moe.h", "rb_common.cuh"}


def test_server_command_line_serves_a_model_folder(tmp_path):
    import urllib.request

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
