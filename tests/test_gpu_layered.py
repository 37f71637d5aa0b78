"""Layered decoders (Dolurax) on the GPU: every kernel against plain math, then the step function, the cache and the engine
against tests/layered_oracle.py in bf16 and in true 32-bit."""
import pytest
import torch

import layered_checks as C
import layered_oracle as O
from rustral_b200.ops import (ScoreRule, distance_slopes, embedding_residual, gemm, head_prep_, residual_norm, scale_softcap_)
from rustral_b200.ops import attention as attn_ops
from rustral_b200.ops import moe as moe_ops
from rustral_b200.ops import paged as paged_ops
from rustral_b200.serve import ServingEngine

pytestmark = [pytest.mark.gpu, pytest.mark.usefixtures("cuda_status")]
BF16, F32 = torch.bfloat16, torch.float32
BOTH = pytest.mark.parametrize("dtype", [BF16, F32], ids=["bf16", "fp32"])


def dev(t, dtype=None):
    return t.to("cuda", dtype or t.dtype)


def close(got, want, tol, what=""):
    got = got.float().cpu()
    assert torch.isfinite(got).all(), what
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-6))
    assert err < tol, (what, err)


def oracle_attention(q, k, v, scale, rule, gate=None):
    """q [L, H, dk] are the last L rows of the keys' positions; fp64 over all keys."""
    S, L = k.shape[0], q.shape[0]
    full = torch.zeros(S, *q.shape[1:])
    full[S - L:] = q
    o = O.attention(full.double(), k.double(), v.double(), scale, rule.softcap, rule.chunk)[S - L:]
    if rule.slopes is None:
        raise ValueError("the plain form always has the distance bias")
    o = o.reshape(L, -1).float()
    return o if gate is None else o * torch.sigmoid(gate)


def qkv(L, S, H, G, dk, dv, seed=0, sharp=1.0):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g).bfloat16().float()
    return (sharp * r(L, H, dk)).bfloat16().float(), r(S, G, dk), r(S, G, dv), r(L, H * dv)


PROMPTS = [  # L, S, heads, kv heads, dk, dv, cap, chunk
    (1, 1, 2, 1, 64, 64, 8.0, 0), (2, 2, 2, 2, 8, 8, 8.0, 16), (130, 130, 4, 2, 96, 64, 0.0, 0), (300, 300, 4, 1, 88, 56, 17.0, 48),
    (257, 700, 2, 1, 128, 128, 15.0, 300), (256, 256, 2, 2, 64, 128, 9.0, 128), (513, 513, 2, 1, 128, 64, 9.0, 256),
    (2, 200, 4, 2, 48, 40, 30.0, 127), (140, 141, 2, 1, 32, 72, 30.0, 1), (600, 1000, 2, 1, 72, 24, 12.0, 129),
    (384, 1024, 1, 1, 112, 104, 12.0, 513), (129, 400, 6, 3, 64, 32, 6.0, 4096), (700, 700, 2, 1, 80, 96, 10.0, 200),
]


@pytest.mark.parametrize("case", PROMPTS, ids=str)
def test_flash_kernel_with_a_score_rule(case):
    L, S, H, G, dk, dv, cap, chunk = case
    q, k, v, gate = qkv(L, S, H, G, dk, dv, sharp=2.0)
    rule = ScoreRule(cap, distance_slopes(H, "cuda"), chunk)
    scale = dk ** -0.5 * 1.3
    pitch = H * dk + H * dv
    z = torch.zeros(L, pitch, dtype=BF16, device="cuda")                   # q and gate inside one packed buffer
    z[:, :H * dk], z[:, H * dk:] = dev(q.reshape(L, -1), BF16), dev(gate, BF16)
    for g in (None, z[:, H * dk:]):
        out = torch.full((1, L, H, dv), 7.0, dtype=BF16, device="cuda")
        assert attn_ops.prompt_supported(z[:, :H * dk], dev(k, BF16).view(S, -1), dev(v, BF16).view(S, -1), dk, dv, rule, g)
        attn_ops.prompt_attention(z[:, :H * dk].view(1, L, H, dk), dev(k, BF16)[None], dev(v, BF16)[None], scale, out, rule, g)
        close(out.view(L, -1), oracle_attention(q, k, v, scale, rule, None if g is None else gate), 1.5e-2, (case, g is not None))


@pytest.mark.parametrize("sharp", [0.1, 1.0, 4.0, 16.0])
def test_flash_kernel_cap_at_small_and_large_scores(sharp):
    """Scores from far below the cap to far above it (the kernel evaluates the cap in two ways)."""
    L, H, dk, dv, cap = 200, 2, 64, 64, 5.0
    q, k, v, _ = qkv(L, L, H, 1, dk, dv, seed=7, sharp=sharp)
    rule = ScoreRule(cap, distance_slopes(H, "cuda"), 90)
    out = torch.empty(1, L, H, dv, dtype=BF16, device="cuda")
    attn_ops.prompt_attention(dev(q, BF16)[None], dev(k, BF16)[None], dev(v, BF16)[None], 0.2, out, rule)
    close(out.view(L, -1), oracle_attention(q, k, v, 0.2, rule), 1.5e-2, sharp)


def paged(k, v, bs, dtype, seed=0):
    """One sequence's keys and values on scattered pages among pages full of other values."""
    S, G, dk = k.shape
    n = -(-S // bs)
    nb = n + 5
    perm = torch.randperm(nb, generator=torch.Generator().manual_seed(seed))[:n]
    kc, vc = torch.full((nb, bs, G, dk), 50.0), torch.full((nb, bs, G, v.shape[2]), 1e4)
    for j in range(S):
        kc[perm[j // bs], j % bs], vc[perm[j // bs], j % bs] = k[j], v[j]
    return dev(kc, dtype), dev(vc, dtype), perm.to(torch.int32)


DECODES = [  # context, heads, kv heads, dk, dv, cap, chunk, page
    (1, 2, 1, 64, 64, 8.0, 0, 16), (17, 4, 2, 96, 56, 18.0, 16, 16), (16, 4, 2, 96, 56, 18.0, 16, 16), (700, 8, 2, 128, 128, 15.0, 0, 16),
    (900, 8, 1, 128, 64, 0.0, 513, 16), (257, 40, 2, 64, 96, 9.0, 256, 4), (333, 4, 4, 48, 40, 9.0, 300, 64), (300, 6, 3, 8, 128, 9.0, 1, 16),
]


@pytest.mark.parametrize("case", DECODES, ids=str)
def test_paged_kernels_with_a_score_rule(case):
    ctx, H, G, dk, dv, cap, chunk, bs = case
    q, k, v, gate = qkv(1, ctx, H, G, dk, dv, seed=ctx, sharp=2.0)
    rule = ScoreRule(cap, distance_slopes(H, "cuda"), chunk)
    scale = dk ** -0.5 * 1.3
    want = oracle_attention(q, k, v, scale, rule, gate)
    short = 1 + ctx // 3                                     # a second, shorter sequence in the same batch
    q2, k2, v2, gate2 = qkv(1, short, H, G, dk, dv, seed=ctx + 1, sharp=2.0)
    want2 = oracle_attention(q2, k2, v2, scale, rule, gate2)
    for dtype in (BF16, F32):
        kc, vc, t1 = paged(k, v, bs, dtype)
        kc2, vc2, t2 = paged(k2, v2, bs, dtype, 1)
        bt = torch.zeros(2, max(len(t1), len(t2)) + 3, dtype=torch.int32)
        bt[0, :len(t1)], bt[1, :len(t2)] = t1, t2 + kc.shape[0]
        kc, vc, bt = torch.cat([kc, kc2]), torch.cat([vc, vc2]), dev(bt)
        qd = dev(torch.cat([q, q2]).view(2, -1), dtype)
        gd = dev(torch.cat([gate, gate2]), dtype)
        rows = paged_ops.paged_attention_rows(qd, kc, vc, bt, torch.arange(2, dtype=torch.int32, device="cuda"),
                                              torch.tensor([ctx - 1, short - 1], device="cuda"), scale, rule, gd)
        close(rows, torch.cat([want, want2]), 1e-2 if dtype == BF16 else 1e-5, ("rows", dtype))
        if dtype == BF16:
            assert paged_ops.decode_supported(qd, dk, dv, rule, gd)
            got = paged_ops.paged_attention_decode(qd, kc, vc, bt, torch.tensor([ctx, short], dtype=torch.int32, device="cuda"),
                                                   scale, rule=rule, gate=gd)
            close(got, torch.cat([want, want2]), 1e-2, "decode")


@pytest.mark.parametrize("i,j,sees", [(127, 64, True), (128, 127, False), (191, 128, True), (192, 191, False), (255, 192, True),
                                      (300, 256, True), (256, 255, False)])
def test_chunk_edges_with_a_key_that_stands_out(i, j, sees):
    """Chunks of 64: prompt kernel, decode kernel and row kernel agree on which far key a query sees."""
    T, H, G, dk, dv = 320, 2, 1, 64, 32
    q, k, v = C.standout_case(i, j, T, H, G, dk, dv)
    rule = ScoreRule(0.0, torch.zeros(H, device="cuda"), 64)
    kc, vc, t = paged(k[:i + 1], v[:i + 1], 16, BF16)
    bt, qi = dev(t)[None].contiguous(), dev(q[i].reshape(1, -1), BF16)
    full = torch.empty(1, T, H, dv, dtype=BF16, device="cuda")
    attn_ops.prompt_attention(dev(q, BF16)[None], dev(k, BF16)[None], dev(v, BF16)[None], 1.0, full, rule)
    got = [full[0, i], paged_ops.paged_attention_decode(qi, kc, vc, bt, torch.tensor([i + 1], dtype=torch.int32, device="cuda"), 1.0, rule=rule)[0].view(H, dv),
           paged_ops.paged_attention_rows(qi, kc, vc, bt, torch.zeros(1, dtype=torch.int32, device="cuda"), torch.tensor([i], device="cuda"), 1.0, rule)[0].view(H, dv)]
    for o in got:
        assert torch.allclose(o.float().cpu(), v[j].expand(H, dv), atol=0.02) == sees
        assert torch.allclose(o.float(), got[0].float(), atol=0.02)


@BOTH
@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 96, 64), (3, 1, 128, 24), (2, 2, 20, 12), (5, 5, 8, 200), (1, 1, 256, 256)])
def test_head_prep(H, G, dk, dv, dtype):
    g = torch.Generator().manual_seed(0)
    T, bs = 37, 4
    p = torch.randn(T, H * dk + G * (dk + dv) + H * dv, generator=g).to(dtype).float()
    first = torch.randn(T, G * dv, generator=g).to(dtype).float()
    qg, kg = torch.randn(dk, generator=g).to(dtype).float(), torch.randn(dk, generator=g).to(dtype).float()
    slots = torch.randperm(60, generator=g)[:T]
    slots[5] = -1
    want, kc, vc = p.clone(), torch.zeros(15, bs, G, dk), torch.zeros(15, bs, G, dv)
    kw = dict(eps=1e-4, slots=slots)
    head_prep_(want, H, G, dk, dv, q_gamma=qg, k_gamma=kg, v_first=first, mix=torch.tensor([0.3]), k_cache=kc, v_cache=vc, **kw)
    got, kd, vd = dev(p, dtype), torch.zeros_like(kc, dtype=dtype, device="cuda"), torch.zeros_like(vc, dtype=dtype, device="cuda")
    head_prep_(got, H, G, dk, dv, q_gamma=dev(qg, dtype), k_gamma=dev(kg, dtype), v_first=dev(first, dtype), mix=torch.tensor([0.3], device="cuda"),
               k_cache=kd, v_cache=vd, eps=1e-4, slots=dev(slots))
    tol = 6e-3 if dtype == BF16 else 1e-5
    close(got, want, tol)
    close(kd, kc, tol)
    close(vd, vc, tol)


@BOTH
@pytest.mark.parametrize("n", [24, 90, 192, 1032, 4096, 8192])
def test_residual_norm(n, dtype):
    g = torch.Generator().manual_seed(n)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    T, k = 19, 3
    y, add, x, gam, bet = r(T * k, n), r(T, n), torch.randn(T, n, generator=g), r(n), r(n)
    slot, w = torch.randperm(T * k, generator=g).to(torch.int32), torch.rand(T, k, generator=g)
    for routed, use_x, rms in ((None, True, False), ((slot, w), True, False), ((slot, w), False, True), (None, False, False)):
        src = y[:T] if routed is None else y
        xw, hw = x.clone(), torch.empty(T, n)
        residual_norm(src, gam, None if rms else bet, 1e-5, rms, x=xw if use_x else None, h=hw, routed=routed, add=add)
        xd, hd = dev(x.clone()), torch.empty(T, n, dtype=dtype, device="cuda")
        residual_norm(dev(src, dtype), dev(gam, dtype), None if rms else dev(bet, dtype), 1e-5, rms, x=xd if use_x else None, h=hd,
                      routed=None if routed is None else (dev(slot), dev(w)), add=dev(add, dtype))
        close(hd, hw, 5e-3 if dtype == BF16 else 1e-5)
        if use_x:
            close(xd, xw, 1e-5)                              # the residual is 32-bit in both


@pytest.mark.parametrize("E,k,groups,keep", [(16, 2, 2, 1), (12, 3, 3, 2), (128, 8, 8, 4), (256, 8, 8, 2), (1, 1, 1, 1), (6, 6, 1, 1), (40, 5, 40, 6), (80, 40, 1, 1), (600, 4, 6, 3)])
def test_router(E, k, groups, keep):
    logits = 2 * torch.randn(133, E, generator=torch.Generator().manual_seed(E))
    iw, ww = moe_ops.route_groups(logits, k, groups, keep)
    ig, wg = moe_ops.route_groups(dev(logits), k, groups, keep)
    assert torch.equal(ig.cpu(), iw)
    close(wg, ww, 1e-5)


@BOTH
def test_expert_products_over_live_rows(dtype):
    g = torch.Generator().manual_seed(3)
    T, d, ff, E, k = 70, 64, 40, 6, 2
    x = torch.randn(T, d, generator=g).to(dtype).float()
    w1, w2 = (torch.randn(E, 2 * ff, d, generator=g) / 8).to(dtype).float(), (torch.randn(E, d, ff, generator=g) / 6).to(dtype).float()
    idx, w = moe_ops.route_groups(torch.randn(T, E, generator=g), k)
    want = torch.zeros(T, d)
    for t in range(T):
        for j in range(k):
            e = int(idx[t, j])
            want[t] += w[t, j] * ((O.silu(x[t] @ w1[e, :ff].T) * (x[t] @ w1[e, ff:].T)) @ w2[e].T)
    pl = moe_ops.plan(dev(idx), E)
    xp = moe_ops.scatter_tokens(dev(x, dtype), pl)
    h = moe_ops.swiglu_rows(moe_ops.grouped_gemm(xp, dev(w1, dtype), pl), pl)
    y = moe_ops.grouped_gemm(h, dev(w2, dtype), pl)
    got = (y[pl.slot_pos.long()].float().view(T, k, d) * dev(w)[:, :, None]).sum(1)
    close(got, want, 2e-2 if dtype == BF16 else 1e-5)


@pytest.mark.parametrize("M,N,K", [(1, 1, 1), (3, 70, 17), (129, 65, 200), (64, 128, 96)])
def test_fp32_product_is_not_rounded(M, N, K):
    g = torch.Generator().manual_seed(M)
    a, b = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g)
    close(gemm(dev(a), dev(b), alpha=0.5), (0.5 * a.double() @ b.double().T).float(), 1e-6)
    with pytest.raises(TypeError):
        gemm(dev(a), dev(b), act="gelu")


@BOTH
def test_embedding_and_logit_cap(dtype):
    t = torch.randn(50, 24, generator=torch.Generator().manual_seed(0)).to(dtype)
    ids = torch.tensor([3, 49, 0, 3])
    x, h = embedding_residual(dev(ids), dev(t))
    assert x.dtype == F32 and h.dtype == dtype and torch.equal(x.cpu(), t[ids].float()) and torch.equal(h.cpu(), t[ids])
    z = 30 * torch.randn(5, 33, generator=torch.Generator().manual_seed(1))
    close(scale_softcap_(dev(z), 2.0, 15.0), 15.0 * torch.tanh(2.0 * z / 15.0), 1e-6)
    close(scale_softcap_(dev(z), 2.0), 2.0 * z, 1e-6)


@BOTH
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_prefill_portions_and_decoding_agree_with_the_plain_model(name, dtype):
    C.check_prefill_portions_and_decode(name, "cuda", dtype)


@BOTH
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_mixed_batches_with_reused_pages(name, dtype):
    C.check_mixed_batch_with_reused_pages(name, "cuda", dtype)


@BOTH
@pytest.mark.parametrize("name", ["varied", "wide"])
def test_long_decoding(name, dtype):
    C.check_long_decoding(name, "cuda", dtype, 330)


def test_greedy_generation_through_the_engine_in_32_bit():
    cfg = C.CONFIGS["wide"]
    w = C.weights(cfg, 6)
    eng = ServingEngine(C.runner(cfg, w, "cuda", F32, blocks=60), max_batch_size=3, prefill_chunk=64)
    prompts = [C.tokens(cfg, n, 20 + n) for n in (5, 170, 33, 1)]
    ids = [eng.submit(p, 8) for p in prompts]
    eng.run_to_completion()
    wd = {k: v.double() for k, v in w.items()}
    for p, rid in zip(prompts, ids):
        assert eng.scheduler.get(rid).generated == O.greedy(cfg, wd, p, 8)
    assert eng.runner.cache.free_blocks == 60


def test_generation_in_bf16_does_not_depend_on_the_batch():
    """The same request alone and beside others, whole and in portions: logits agree beyond rounding, so greedy tokens do."""
    cfg = C.CONFIGS["wide"]
    w = C.weights(cfg, 6)
    prompts = [C.tokens(cfg, n, 50 + n) for n in (60, 7, 161)]
    alone = [ServingEngine(C.runner(cfg, w, "cuda", BF16, blocks=60)).generate(p, 4) for p in prompts]
    eng = ServingEngine(C.runner(cfg, w, "cuda", BF16, blocks=60), max_batch_size=4, prefill_chunk=50)
    ids = [eng.submit(p, 4) for p in prompts]
    eng.run_to_completion()
    same = sum(eng.scheduler.get(r).generated[0] == a[0] for r, a in zip(ids, alone))
    assert same >= 2
