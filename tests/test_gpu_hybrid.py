"""Hybrid decoders (Vafodra) on the GPU: every kernel against plain math, then the step function, the cache with its state slots and
the engine against tests/hybrid_oracle.py in bf16 and in true 32-bit."""
import pytest
import torch

import hybrid_checks as C
import hybrid_oracle as O
from rustral_b200.ops import (ScoreRule, Segments, delta_rule, embedding_residual, gated_norm, head_prep_, short_conv, state_space,
                              stream_update)
from rustral_b200.ops import attention as attn_ops
from rustral_b200.ops import paged as paged_ops
from rustral_b200.ops.moe import swiglu_rows
from rustral_b200.ops.recurrent import _span, up4
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


def qkv(L, S, H, G, dk, dv, seed=0, sharp=1.0):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g).bfloat16().float()
    return (sharp * r(L, H, dk)).bfloat16().float(), r(S, G, dk), r(S, G, dv), torch.randn(L, H, generator=g)


def oracle(q, k, v, scale, rule, gate=None):
    """q [L, H, dk] are the last L rows of the keys' positions."""
    S, L = k.shape[0], q.shape[0]
    full = torch.zeros(S, *q.shape[1:])
    full[S - L:] = q
    o = O.attention(full.double(), k.double(), v.double(), scale, rule.window, rule.keep_first, rule.sink)[S - L:].float()
    return (o if gate is None else o * torch.sigmoid(gate)[:, :, None]).reshape(L, -1)


PROMPTS = [  # L, S, heads, kv heads, dk, dv, window, kept, sink
    (1, 1, 2, 1, 64, 64, 8, 0, True), (2, 2, 2, 2, 8, 8, 1, 0, True), (130, 130, 4, 2, 96, 64, 0, 0, True), (300, 300, 4, 1, 88, 56, 48, 3, True),
    (257, 700, 2, 1, 128, 128, 300, 4, True), (256, 256, 2, 2, 64, 128, 128, 0, True), (513, 513, 2, 1, 128, 64, 129, 1, False),
    (2, 200, 4, 2, 48, 40, 63, 7, True), (140, 141, 2, 1, 32, 72, 1, 0, True), (600, 1000, 2, 1, 72, 24, 129, 128, True),
    (384, 1024, 1, 1, 112, 104, 256, 130, True), (129, 900, 6, 3, 64, 32, 4096, 4, True), (700, 900, 2, 1, 80, 96, 37, 300, True),
    (260, 900, 2, 2, 64, 64, 500, 0, False), (64, 640, 2, 1, 64, 64, 64, 2, True),
]


@pytest.mark.parametrize("case", PROMPTS, ids=str)
def test_flash_kernel_with_a_window(case):
    L, S, H, G, dk, dv, window, keep, sink = case
    q, k, v, gate = qkv(L, S, H, G, dk, dv, sharp=2.0)
    rule = ScoreRule(window=window, keep_first=keep, sink=sink)
    scale = dk ** -0.5 * 1.3
    kept, first = rule.key_ranges(S - L)
    keys = [*range(kept), *range(first, S)]                                # what the portion gathers ...
    for idx in (list(range(S)), keys):                                      # ... gives the same as all keys
        for g in (None, gate):
            out = torch.full((1, L, H, dv), 7.0, dtype=BF16, device="cuda")
            qd, kd, vd = dev(q, BF16)[None], dev(k[idx], BF16)[None], dev(v[idx], BF16)[None]
            assert attn_ops.prompt_supported(qd[0].view(L, -1), kd[0].view(len(idx), -1), vd[0].view(len(idx), -1), dk, dv, rule)
            attn_ops.prompt_attention(qd, kd, vd, scale, out, rule, head_gate=None if g is None else dev(g))
            close(out.view(L, -1), oracle(q, k, v, scale, rule, g), 1.5e-2, (case, len(idx), g is not None))


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


DECODES = [  # context, heads, kv heads, dk, dv, window, kept, sink, page
    (1, 2, 1, 64, 64, 8, 0, True, 16), (17, 4, 2, 96, 56, 16, 1, True, 16), (16, 4, 2, 96, 56, 16, 1, True, 16), (700, 8, 2, 128, 128, 0, 0, True, 16),
    (900, 8, 1, 128, 64, 513, 4, True, 16), (257, 40, 2, 64, 96, 256, 0, False, 4), (333, 4, 4, 48, 40, 100, 40, True, 64), (300, 6, 3, 8, 128, 1, 0, True, 16),
    (600, 6, 3, 64, 64, 100, 300, True, 16), (520, 2, 2, 64, 64, 252, 5, True, 16), (300, 6, 3, 20, 12, 30, 2, True, 16),
]


@pytest.mark.parametrize("case", DECODES, ids=str)
def test_paged_kernels_with_a_window(case):
    ctx, H, G, dk, dv, window, keep, sink, bs = case
    rule = ScoreRule(window=window, keep_first=keep, sink=sink)
    scale = dk ** -0.5 * 1.3
    short = 1 + ctx // 3                                     # a second, shorter sequence in the same batch
    rows = [qkv(1, n, H, G, dk, dv, seed=n, sharp=2.0) for n in (ctx, short)]
    want = torch.cat([oracle(q, k, v, scale, rule, gate) for q, k, v, gate in rows])
    for dtype in (BF16, F32):
        (kc, vc, t1), (kc2, vc2, t2) = (paged(r[1], r[2], bs, dtype, i) for i, r in enumerate(rows))
        bt = torch.zeros(2, max(len(t1), len(t2)) + 3, dtype=torch.int32)
        bt[0, :len(t1)], bt[1, :len(t2)] = t1, t2 + kc.shape[0]
        kc, vc, bt = torch.cat([kc, kc2]), torch.cat([vc, vc2]), dev(bt)
        qd = dev(torch.cat([r[0] for r in rows]).view(2, -1), dtype)
        gd = torch.zeros(2, H + 3, device="cuda")
        gd[:, 1:H + 1] = dev(torch.cat([r[3] for r in rows]))                # gates inside a wider buffer
        gd = gd[:, 1:H + 1]
        got = paged_ops.paged_attention_rows(qd, kc, vc, bt, torch.arange(2, dtype=torch.int32, device="cuda"),
                                             torch.tensor([ctx - 1, short - 1], device="cuda"), scale, rule, head_gate=gd)
        close(got, want, 1e-2 if dtype == BF16 else 1e-5, ("rows", dtype))
        if dtype == BF16 and paged_ops.decode_supported(qd, dk, dv, rule):
            got = paged_ops.paged_attention_decode(qd, kc, vc, bt, torch.tensor([ctx, short], dtype=torch.int32, device="cuda"),
                                                   scale, rule=rule, head_gate=gd)
            close(got, want, 1e-2, "decode")


@pytest.mark.parametrize("i,j,sees", [(127, 64, True), (128, 64, False), (191, 128, True), (300, 237, True), (300, 236, False), (300, 2, True),
                                      (300, 3, False), (319, 0, True), (63, 0, True), (66, 3, True), (67, 3, False)])
def test_window_edges_with_a_key_that_stands_out(i, j, sees):
    """Windows of 64 with three kept tokens: prompt kernel, decode kernel and row kernel agree on which far key a query sees."""
    T, H, G, dk, dv = 320, 2, 1, 64, 32
    q, k, v = C.standout_case(i, j, T, H, G, dk, dv)
    rule = ScoreRule(window=64, keep_first=3, sink=True)
    kc, vc, t = paged(k[:i + 1], v[:i + 1], 16, BF16)
    bt, qi = dev(t)[None].contiguous(), dev(q[i].reshape(1, -1), BF16)
    full = torch.empty(1, T, H, dv, dtype=BF16, device="cuda")
    attn_ops.prompt_attention(dev(q, BF16)[None], dev(k, BF16)[None], dev(v, BF16)[None], 1.0, full, rule)
    got = [full[0, i], paged_ops.paged_attention_decode(qi, kc, vc, bt, torch.tensor([i + 1], dtype=torch.int32, device="cuda"), 1.0, rule=rule)[0].view(H, dv),
           paged_ops.paged_attention_rows(qi, kc, vc, bt, torch.zeros(1, dtype=torch.int32, device="cuda"), torch.tensor([i], device="cuda"), 1.0, rule)[0].view(H, dv)]
    for o in got:
        assert torch.allclose(o.float().cpu(), v[j].expand(H, dv), atol=0.02) == sees == O.visible(i, j, 64, 3)
        assert torch.allclose(o.float(), got[0].float(), atol=0.02)


SEGMENTS = {"one": [(0, 150, 1, 0)], "several": [(0, 2, 3, 0), (2, 64, 0, 5), (66, 1, 2, 0), (67, 1, 4, 9), (68, 65, 1, 0), (133, 17, 5, 3)],
            "decode": [(i, 1, (5 * i + 2) % 7, i % 3) for i in range(7)], "long": [(0, 700, 2, 3), (700, 330, 0, 0)]}


@BOTH
@pytest.mark.parametrize("name", sorted(SEGMENTS))
@pytest.mark.parametrize("channels,taps", [(24, 4), (136, 2), (9, 3), (40, 7), (16, 1)])
def test_short_conv(channels, taps, name, dtype):
    segs = SEGMENTS[name]
    T = sum(s[1] for s in segs)
    g = torch.Generator().manual_seed(taps)
    x, w, b = torch.randn(T, channels + 8, generator=g).to(dtype), torch.randn(channels, taps, generator=g), torch.randn(channels, generator=g)
    state = torch.randn(8, taps - 1, channels, generator=g).to(dtype)
    for bias in (b, None):
        sw, sd = state.clone().float(), dev(state)
        want = short_conv(x[:, 4:4 + channels].float(), w, bias, sw, Segments.of(segs, "cpu"))
        got = short_conv(dev(x)[:, 4:4 + channels], dev(w), None if bias is None else dev(bias), sd, Segments.of(segs, "cuda"))
        close(got, want, 5e-3 if dtype == BF16 else 1e-5)
        assert torch.equal(sd.cpu().float(), sw)             # inputs, kept as they are


SSM = [  # heads, groups, vdim, state, shift of the logarithm of the decay rate
    (2, 1, 64, 128, 0.0), (4, 2, 56, 40, -2.0), (2, 2, 128, 64, 1.5), (3, 1, 40, 24, -4.0), (2, 1, 72, 104, 0.0), (2, 1, 20, 12, 0.0), (1, 1, 8, 200, 0.0),
]


@BOTH
@pytest.mark.parametrize("name", sorted(SEGMENTS))
@pytest.mark.parametrize("case", SSM, ids=str)
def test_state_space(case, name, dtype):
    H, G, P, N, shift = case
    segs = SEGMENTS[name]
    T = sum(s[1] for s in segs)
    g = torch.Generator().manual_seed(H * P + N)
    r = lambda *s: torch.randn(*s, generator=g)
    xbc, dt, state = r(T, H * P + 2 * G * N).to(dtype), r(T, H), r(8, H, N, up4(P))
    kw = dict(dt_bias=r(H) - 1, a_log=r(H) + shift, D=r(H))
    sw, sd = state.clone(), dev(state)
    args = dict(heads=H, groups=G, vdim=P, n=N)
    want = state_space(xbc.float(), dt, state=sw, seg=Segments.of(segs, "cpu"), **kw, **args)
    got = state_space(dev(xbc), dev(dt), state=sd, seg=Segments.of(segs, "cuda"), **{k: dev(v) for k, v in kw.items()}, **args)
    close(got, want, 1e-2 if dtype == BF16 else 1e-5)
    close(sd[..., :P], sw[..., :P], 2e-5)                    # the state is 32-bit in both


def test_state_space_spans_of_a_long_prompt():
    """Cut into spans that run side by side, whatever their number: y and the state are those of one span."""
    H, G, P, N = 2, 1, 64, 64
    g = torch.Generator().manual_seed(5)
    r = lambda *s: torch.randn(*s, generator=g)
    segs = [(0, 900, 1, 7), (900, 515, 0, 0)]
    xbc, dt, state = r(1415, H * P + 2 * G * N).to(BF16), r(1415, H), r(2, H, N, P)
    kw = dict(dt_bias=r(H) - 3, a_log=r(H) - 3, D=r(H), heads=H, groups=G, vdim=P, n=N)
    sw = state.clone()
    want = state_space(xbc.float(), dt, state=sw, seg=Segments.of(segs, "cpu"), **kw)
    for size in (128, 256, 512, 1024):
        import rustral_b200.ops.recurrent as rc
        seg, sd = Segments.of(segs, "cuda"), dev(state)
        keep, rc._span = rc._span, lambda *a: size
        try:
            got = state_space(dev(xbc), dev(dt), state=sd, seg=seg, **{k: dev(v) if torch.is_tensor(v) else v for k, v in kw.items()})
        finally:
            rc._span = keep
        close(got, want, 1e-2, size)
        close(sd, sw, 2e-5, size)
    assert _span(Segments.of([(0, 64, 0, 0)], "cpu"), 4) >= 64 and _span(Segments.of([(0, 8192, 0, 0)], "cpu"), 64) % 128 == 0


DELTA = [  # heads, kv heads, dk, dv, shift of the logarithm of the decay rate
    (2, 1, 128, 64, 0.0), (4, 2, 40, 72, -2.0), (2, 2, 64, 128, 1.5), (3, 3, 24, 40, -4.0), (2, 1, 104, 136, -6.0), (2, 1, 20, 12, 0.0), (1, 1, 200, 8, 0.0),
]


@BOTH
@pytest.mark.parametrize("name", sorted(SEGMENTS))
@pytest.mark.parametrize("case", DELTA, ids=str)
def test_delta_rule(case, name, dtype):
    H, G, dk, dv, shift = case
    segs = SEGMENTS[name]
    T = sum(s[1] for s in segs)
    g = torch.Generator().manual_seed(H * dk + dv)
    r = lambda *s: torch.randn(*s, generator=g)
    qkv_, ab, state = r(T, 2 * G * dk + H * dv).to(dtype), 2 * r(T, 2 * H), r(8, H, dk, up4(dv))
    if name == "one":
        qkv_[:, G * dk:2 * G * dk] = (qkv_[:1, G * dk:2 * G * dk].float() + 0.3 * r(T, G * dk)).to(dtype)     # keys that are much alike
    kw = dict(dt_bias=r(H) - 1, a_log=r(H) + shift)
    args = dict(heads=H, kv_heads=G, dk=dk, dv=dv)
    sw, sd, abd = state.clone(), dev(state), dev(ab)
    want = delta_rule(qkv_.float(), ab[:, :H], ab[:, H:], state=sw, seg=Segments.of(segs, "cpu"), **kw, **args)
    out = torch.full((T, H * dv + 8), 3.0, dtype=dtype, device="cuda")
    delta_rule(dev(qkv_), abd[:, :H], abd[:, H:], state=sd, seg=Segments.of(segs, "cuda"), out=out[:, :H * dv], **{k: dev(v) for k, v in kw.items()}, **args)
    close(out[:, :H * dv], want, 1e-2 if dtype == BF16 else 2e-5)
    close(sd[..., :dv], sw[..., :dv], 5e-5)
    assert bool((out[:, H * dv:] == 3.0).all())


def test_portions_of_a_prompt_give_the_same_state():
    """Chunked kernels, scan kernels and any mixture of them leave the same states behind."""
    g = torch.Generator().manual_seed(3)
    r = lambda *s: torch.randn(*s, generator=g)
    H, G, d, T = 4, 2, 64, 300
    qkv_, ab, xbc = dev(r(T, 2 * G * d + H * d), BF16), dev(r(T, 2 * H)), dev(r(T, H * d + 2 * G * d), BF16)
    bias, a_log, D = dev(r(H) - 2), dev(r(H) - 2), dev(r(H))
    states = []
    for cuts in ([], [64, 128], [1, 2, 4, 70, 71, 200], list(range(1, T))):
        s1, s2 = torch.full((1, H, d, d), 1e4, device="cuda"), torch.full((1, H, d, d), 1e4, device="cuda")
        lo = 0
        for hi in [*cuts, T]:
            seg = Segments.of([(0, hi - lo, 0, lo)], "cuda")
            delta_rule(qkv_[lo:hi], ab[lo:hi, :H], ab[lo:hi, H:], dt_bias=bias, a_log=a_log, state=s1, heads=H, kv_heads=G, dk=d, dv=d, seg=seg)
            state_space(xbc[lo:hi], ab[lo:hi, :H], dt_bias=bias, a_log=a_log, D=D, state=s2, heads=H, groups=G, vdim=d, n=d, seg=seg)
            lo = hi
        states.append((s1, s2))
    for a, b in states[1:]:
        close(a, states[0][0].cpu(), 5e-5)
        close(b, states[0][1].cpu(), 2e-5)


@BOTH
@pytest.mark.parametrize("n,parts", [(24, 3), (96, 1), (90, 5), (1024, 8), (4096, 1), (4096, 32), (8200, 1), (520, 4), (2048, 32), (1536, 2), (3000, 1), (448, 2)])
def test_gated_norm(n, parts, dtype):
    g = torch.Generator().manual_seed(n)
    y, z, w = torch.randn(19, n, generator=g).to(dtype), torch.randn(19, n + 8, generator=g).to(dtype), torch.randn(n, generator=g)
    z = z[:, 8:]
    tol = 6e-3 if dtype == BF16 else 1e-5
    close(gated_norm(dev(y), dev(z), dev(w), parts, 1e-3, True), O.gated_group_norm(y.float(), z.float(), w, parts, 1e-3), tol)
    part = w[:n // parts]
    want = (O.rms_norm(y.float().view(19, parts, -1), part, 1e-3)).reshape(19, n) * O.silu(z.float())
    yd = dev(y)
    close(gated_norm(yd, dev(z), dev(part), parts, 1e-3, False, out=yd), want, tol)      # in place


@BOTH
@pytest.mark.parametrize("n", [24, 90, 192, 1032, 4096])
def test_stream_update(n, dtype):
    g = torch.Generator().manual_seed(n)
    r = lambda *s: torch.randn(*s, generator=g)
    T = 19
    x, a, b, c = r(T, n), r(T, n).to(dtype), r(T, n).to(dtype), r(T, n).to(dtype)
    wa, wb, gam, bet, alpha = r(n), r(n), r(n), r(n), torch.tensor([0.7])
    dyt = (dev(gam), dev(bet), dev(alpha))
    for src in ("abc", "ab", "c", ""):
        want = x.clone()
        kw = {}
        if "a" in src:
            want = want + 0.3 * 0.5 * (O.rms_norm(a.float(), wa, 1e-3) + O.rms_norm(b.float(), wb, 1e-3))
            kw.update(a=dev(a), wa=dev(wa), b=dev(b), wb=dev(wb))
        if "c" in src:
            want = want + 0.3 * c.float()
            kw.update(c=dev(c))
        xd, h = dev(x.clone()), torch.empty(T, n, dtype=dtype, device="cuda")
        stream_update(xd, normed=0.5, mult=0.3, eps=1e-3, dyt=dyt, h=h, **kw)
        close(xd, want, 1e-5, src)                            # the residual is 32-bit in both
        close(h, O.dynamic_tanh(want, alpha, gam, bet), 5e-3 if dtype == BF16 else 1e-5, src)


@BOTH
def test_embedding_scale_relu_gate_and_append(dtype):
    t = torch.randn(50, 24, generator=torch.Generator().manual_seed(0)).to(dtype)
    ids = torch.tensor([3, 49, 0, 3])
    x, h = embedding_residual(dev(ids), dev(t), 2.5, want_h=False)
    assert h is None and torch.equal(x.cpu(), t[ids].float() * 2.5)
    x, h = embedding_residual(dev(ids), dev(t), 2.5)
    assert h.dtype == dtype and torch.equal(h.cpu(), (t[ids].float() * 2.5).to(dtype))
    gu, out = torch.randn(33, 80, generator=torch.Generator().manual_seed(1)).to(dtype), torch.zeros(33, 64, dtype=dtype, device="cuda")
    swiglu_rows(dev(gu)[:, 16:64], act="relu", out=out[:, 8:32])
    close(out[:, 8:32], torch.relu(gu[:, 16:40].float()) * gu[:, 40:64].float(), 5e-3 if dtype == BF16 else 1e-6)
    assert float(out[:, :8].abs().max()) == float(out[:, 32:].abs().max()) == 0
    p = torch.randn(5, 40, generator=torch.Generator().manual_seed(2)).to(dtype)
    kc, vc = torch.zeros(2, 4, 2, 4, dtype=dtype, device="cuda"), torch.zeros(2, 4, 2, 8, dtype=dtype, device="cuda")
    pd = dev(p)
    head_prep_(pd, 4, 2, 4, 8, k_cache=kc, v_cache=vc, slots=torch.tensor([7, -1, 0, 3, 5], device="cuda"))       # no norm: append only
    assert torch.equal(pd.cpu(), p) and torch.equal(kc.view(8, 8)[[7, 0, 3, 5]].cpu(), p[[0, 2, 3, 4], 16:24])
    assert torch.equal(vc.view(8, 16)[[7, 0, 3, 5]].cpu(), p[[0, 2, 3, 4], 24:40]) and float(kc.view(8, 8)[[1, 2, 4, 6]].abs().max()) == 0


@BOTH
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_prefill_portions_and_decoding_agree_with_the_plain_model(name, dtype):
    C.check_prefill_portions_and_decode(name, "cuda", dtype)


@BOTH
def test_long_prompt_in_portions(dtype):
    """A prompt of several windows, tiles and chunks of the kernels, cut at and around their edges."""
    C.check_prefill_portions_and_decode("wide", "cuda", dtype, 400, {"whole": [], "around tiles": [63, 64, 66, 128, 129, 191, 256, 320], "halves": [200],
                                                                     "kept edge": [130, 132, 280, 281, 283]})


@BOTH
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_mixed_batches_with_reused_pages_and_slots(name, dtype):
    C.check_mixed_batch_with_reused_pages_and_slots(name, "cuda", dtype)


@BOTH
@pytest.mark.parametrize("name", ["varied", "wide"])
def test_long_decoding(name, dtype):
    C.check_long_decoding(name, "cuda", dtype, 330 if name == "wide" else 200)


def test_greedy_generation_through_the_engine_in_32_bit():
    cfg = C.CONFIGS["wide"]
    w = C.weights(cfg, 6)
    r = C.runner(cfg, w, "cuda", F32, blocks=60, slots=2)
    C.poison(r)
    eng = ServingEngine(r, max_batch_size=3, prefill_chunk=64)
    prompts = [C.tokens(cfg, n, 20 + n) for n in (5, 170, 33, 1)]
    ids = [eng.submit(p, 8) for p in prompts]
    eng.run_to_completion()
    wd = {k: v.double() for k, v in w.items()}
    for p, rid in zip(prompts, ids):
        assert eng.scheduler.get(rid).generated == O.greedy(cfg, wd, p, 8)
    assert r.cache.free_blocks == 60 and r.cache.free_slots == 2


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
