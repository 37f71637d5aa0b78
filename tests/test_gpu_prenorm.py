"""Pre-norm decoders (Seredra) on the GPU: every kernel against plain math, then the step function, the cache and the engine against
tests/prenorm_oracle.py in bf16 and in true 32-bit."""
import pytest
import torch

import prenorm_checks as C
import prenorm_oracle as O
from rustral_b200.models.layered import RotarySpec
from rustral_b200.ops import (ScoreRule, Segments, gated_norm, head_prep_, residual_norm, rotary_table, row_prep_, selective_scan, short_conv, state_space)
from rustral_b200.ops import attention as attn_ops
from rustral_b200.ops import moe as moe_ops
from rustral_b200.ops import paged as paged_ops
from rustral_b200.serve import ServingEngine

pytestmark = [pytest.mark.gpu, pytest.mark.usefixtures("cuda_status")]
BF16, F32 = torch.bfloat16, torch.float32
BOTH = pytest.mark.parametrize("dtype", [BF16, F32], ids=["bf16", "fp32"])


def dev(t, dtype=None):
    return t.to("cuda", dtype or t.dtype)


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def close(got, want, tol, what=""):
    got = got.float().cpu()
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-6))
    assert err < tol, (what, err)


def table_of(rot, pos):
    spec = RotarySpec.from_json(rot, True)
    return rotary_table(pos.cuda(), torch.tensor(spec.frequencies(), dtype=torch.float64, device="cuda"), spec.magnitude)


def turned(x3, pos, rot):
    return O.rotate(x3.double(), pos, rot).float()


# ---- queries, keys, values ---------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("keys", [True, False])
@pytest.mark.parametrize("normed", [True, False])
@pytest.mark.parametrize("H,G,dk,dims", [(4, 2, 64, 64), (6, 2, 104, 32), (2, 2, 128, 128), (4, 1, 24, 16), (3, 3, 20, 6), (2, 1, 40, 8), (1, 1, 13, 12), (4, 2, 200, 48),
                                         (3, 1, 96, 2), (2, 1, 136, 136), (2, 2, 520, 512), (2, 1, 1040, 16)])
def test_head_prep_with_halves(H, G, dk, dims, normed, keys, dtype):
    T = 9
    rot, pos = dict(dims=dims, base=900.0), torch.arange(T) * 37
    p = rnd(T, (H + 2 * G) * dk + 8, seed=dk).to(dtype)
    gq, gk = (rnd(dk, seed=1).to(dtype), rnd(dk, seed=2).to(dtype)) if normed else (None, None)
    slots = torch.tensor([11, 0, 3, -1, 5, 6, 7, 8, 1])
    ov = (H + G) * dk
    q, k = p[:, :H * dk].float().reshape(T, H, dk), p[:, H * dk:ov].float().reshape(T, G, dk)
    v = p[:, H * dk:ov] if keys else p[:, ov:ov + G * dk]
    if normed:
        q, k = O.unit_rms(q, 1e-3) * gq.float(), O.unit_rms(k, 1e-3) * gk.float()
    want_q, want_k = turned(q, pos, rot), turned(k, pos, rot)
    kc, vc, pd = torch.zeros(3, 4, G, dk, dtype=dtype, device="cuda"), torch.zeros(3, 4, G, dk, dtype=dtype, device="cuda"), dev(p)
    head_prep_(pd, H, G, dk, dk, q_gamma=None if gq is None else dev(gq), k_gamma=None if gk is None else dev(gk), eps=1e-3, k_cache=kc, v_cache=vc,
               slots=dev(slots), rot=table_of(rot, pos), half=True, values_are_keys=keys)
    tol, keep = 6e-3 if dtype == BF16 else 1e-5, slots >= 0
    close(pd[:, :H * dk].view(T, H, dk), want_q, tol)
    close(pd[:, H * dk:ov].view(T, G, dk), want_k, tol)
    close(kc.view(12, G, dk)[dev(slots[keep])], want_k[keep], tol)
    assert torch.equal(vc.view(12, G * dk)[dev(slots[keep])].cpu(), v[keep]) and torch.equal(pd[:, ov:ov + G * dk].cpu(), v)
    assert torch.equal(pd[:, ov + G * dk:].cpu(), p[:, ov + G * dk:]) and float(kc.view(12, -1)[[2, 4, 9, 10]].abs().max()) == 0


@BOTH
@pytest.mark.parametrize("H,dk,dims", [(2, 32, 32), (3, 24, 8), (5, 12, 10), (1, 144, 144)])
def test_rotation_with_key_scale_behind_other_columns(H, dk, dims, dtype):
    T, nv = 7, 16
    rot, pos = dict(dims=dims, base=700.0), torch.tensor([0, 5, 90, 3, 3, 1000, 7])
    p = rnd(T, nv + 2 * H * dk + 8).to(dtype)
    pd = dev(p)
    head_prep_(pd, H, H, dk, dk, rot=table_of(rot, pos), half=True, k_scale=dk ** -0.5, q_col=nv + H * dk, k_col=nv)
    want = p.float().clone()
    want[:, nv:nv + H * dk] = dk ** -0.5 * turned(want[:, nv:nv + H * dk].reshape(T, H, dk), pos, rot).reshape(T, -1)
    want[:, nv + H * dk:nv + 2 * H * dk] = turned(want[:, nv + H * dk:nv + 2 * H * dk].reshape(T, H, dk), pos, rot).reshape(T, -1)
    close(pd, want, 5e-3 if dtype == BF16 else 1e-5)
    assert torch.equal(pd[:, :nv].cpu(), p[:, :nv]) and torch.equal(pd[:, -8:].cpu(), p[:, -8:])


@BOTH
@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 64, 64), (6, 3, 24, 40), (1, 1, 8, 8), (6, 3, 13, 11), (32, 8, 128, 128), (64, 16, 128, 128), (3, 0, 40, 16), (5, 0, 7, 3), (80, 60, 136, 8)])
@pytest.mark.parametrize("every", [0, 1, 50])
def test_row_prep(H, G, dk, dv, every, dtype):
    T, nq, nk, nv = 9, H * dk, G * dk, G * dv
    p, gq, gk = rnd(T, nq + nk + nv + 8, seed=dk).to(dtype), rnd(nq, seed=1), rnd(max(nk, 1), seed=2)
    pos, slots = torch.tensor([0, 1, 48, 49, 50, 98, 99, 10 ** 6, 7]), torch.tensor([11, 0, 3, -1, 5, 6, 7, 8, 1])
    want = p.float().clone()
    want[:, :nq] = O.unit_rms(want[:, :nq], 1e-3) * gq
    if every:
        want[:, :nq] *= O.temperature(pos, 0.4, every).float()[:, None]
    want[:, nq:nq + nk] = O.unit_rms(want[:, nq:nq + nk], 1e-3) * gk[:nk]
    kc, vc = (torch.zeros(3, 4, max(G, 1), s, dtype=dtype, device="cuda") for s in (dk, dv))
    pd = dev(p)
    row_prep_(pd, H, G, dk, dv, q_gamma=dev(gq), k_gamma=dev(gk) if G else None, eps=1e-3, pos=dev(pos), temp_coef=0.4, temp_every=every, k_cache=kc, v_cache=vc,
              slots=dev(slots))
    close(pd, want, 6e-3 if dtype == BF16 else 1e-5)
    if G:
        keep = slots >= 0
        assert torch.equal(kc.view(12, -1)[dev(slots[keep])], pd[dev(keep)][:, nq:nq + nk]) and torch.equal(vc.view(12, -1)[dev(slots[keep])].cpu(), p[keep][:, nq + nk:nq + nk + nv])
        assert float(kc.view(12, -1)[[2, 4, 9, 10]].abs().max()) == 0


# ---- attention -----------------------------------------------------------------------------------------------------------
def want_attention(q, k, v, scale, rule):
    S, L = k.shape[0], q.shape[0]
    full = torch.zeros(S, *q.shape[1:])
    full[S - L:] = q
    r1, r2 = (None, None) if rule.log_rate is None else (rule.log_amount.double(), rule.log_rate.double())
    return rule.out_scale * O.attend(full.double(), k.double(), v.double(), scale, rule.softcap, r1, r2)[S - L:].float().reshape(L, -1)


def on_gpu(rule):
    return ScoreRule(softcap=rule.softcap, out_scale=rule.out_scale, log_amount=None if rule.log_rate is None else dev(rule.log_amount),
                     log_rate=None if rule.log_rate is None else dev(rule.log_rate))


def paged(kv, bs, dtype, seed=0):
    """One sequence's keys or values on scattered pages among pages full of other values."""
    S = kv.shape[0]
    n = -(-S // bs)
    perm = torch.randperm(n + 5, generator=torch.Generator().manual_seed(seed))[:n]
    c = torch.full((n + 5, bs, *kv.shape[1:]), 1e4)
    for j in range(S):
        c[perm[j // bs], j % bs] = kv[j]
    return dev(c, dtype), dev(perm.to(torch.int32))[None].contiguous()


RATES = {"steep": 3.0, "usual": 0.2, "slow": 0.001, "none": 0.0}
LOGS = [  # rows, keys, heads, kv heads, dk, dv, cap
    (1, 1, 2, 1, 64, 64, 0.0), (130, 130, 6, 2, 88, 88, 0.0), (300, 300, 4, 1, 88, 56, 5.0), (257, 900, 2, 1, 128, 128, 0.0), (513, 1300, 2, 1, 128, 64, 0.0),
    (2, 700, 4, 2, 48, 40, 9.0), (140, 141, 2, 1, 32, 72, 0.0), (40, 1000, 3, 3, 64, 128, 0.0),
]


@pytest.mark.parametrize("rate", RATES)
@pytest.mark.parametrize("case", LOGS, ids=str)
def test_logarithmic_bias(case, rate):
    """Prompt, decode and row kernels; the prompt kernel takes logarithms near the diagonal and a series further away."""
    L, S, H, G, dk, dv, cap = case
    r = lambda *s, seed: rnd(*s, seed=seed).bfloat16().float()
    q, k, v = (2 * r(L, H, dk, seed=1)).bfloat16().float(), r(S, G, dk, seed=2), r(S, G, dv, seed=3)
    rule = ScoreRule(softcap=cap, out_scale=0.6, log_amount=0.2 + rnd(H, seed=4).abs(), log_rate=RATES[rate] * (0.5 + torch.rand(H, generator=torch.Generator().manual_seed(5))))
    scale = 1.3 * dk ** -0.5
    want, rd = want_attention(q, k, v, scale, rule), on_gpu(rule)
    out = torch.full((1, L, H, dv), 7.0, dtype=BF16, device="cuda")
    assert attn_ops.prompt_supported(dev(q, BF16).view(L, -1), dev(k, BF16).view(S, -1), dev(v, BF16).view(S, -1), dk, dv, rd)
    attn_ops.prompt_attention(dev(q, BF16)[None], dev(k, BF16)[None], dev(v, BF16)[None], scale, out, rd)
    close(out.view(L, -1), want, 1.5e-2, "prompt")
    for dtype in (BF16, F32):
        (kc, bt), (vc, _) = paged(k, 16, dtype), paged(v, 16, dtype)
        rows = paged_ops.paged_attention_rows(dev(q, dtype).view(L, -1), kc, vc, bt, torch.zeros(L, dtype=torch.int32, device="cuda"),
                                              torch.arange(S - L, S, device="cuda"), scale, rd)
        close(rows, want, 1e-2 if dtype == BF16 else 1e-5, "rows")
        if dtype == BF16:
            n = min(L, 4)
            ctx = torch.arange(S - n + 1, S + 1, dtype=torch.int32, device="cuda")
            got = paged_ops.paged_attention_decode(dev(q[L - n:], dtype).reshape(n, -1), kc, vc, bt.expand(n, -1).contiguous(), ctx, scale, rule=rd)
            close(got, want[L - n:], 1e-2, "decode")


def test_logarithmic_bias_of_the_prompt_kernel_is_exact():
    """With zero queries the weights are the bias alone, (1 + r2 d)^(-r1) over their sum: in every tile, near and far."""
    S, H = 1500, 2
    r1, r2 = torch.tensor([0.7, 2.0]), torch.tensor([0.9, 0.03])
    q, k = torch.zeros(S, H, 64), rnd(S, H, 64)
    v = torch.zeros(S, H, 64)
    for j in range(0, S, 32):
        v[j, :, j // 32] = 1.0                                         # one column per marked key
    out = torch.empty(1, S, H, 64, dtype=BF16, device="cuda")
    attn_ops.prompt_attention(dev(q, BF16)[None], dev(k, BF16)[None], dev(v, BF16)[None], 1.0, out, ScoreRule(log_amount=dev(r1), log_rate=dev(r2)))
    o, d = out[0].float().cpu(), torch.arange(S, dtype=torch.float64)
    for i in (0, 1, 127, 128, 300, 511, 777, 1024, 1499):
        for h in range(H):
            w = (1 + r2[h].double() * d[:i + 1]) ** -r1[h].double()
            w = (w / w.sum()).flip(0)                                    # by key
            for j in range(0, i + 1, 32):
                assert float(o[i, h, j // 32]) == pytest.approx(float(w[j]), rel=1.2e-2, abs=1e-6), (i, h, j)


@pytest.mark.parametrize("far", [0, 1, 127, 128, 255, 256, 400, 511, 512, 639])
def test_a_key_that_stands_out_is_found_at_any_distance(far):
    S, H, G, dk, dv = 640, 4, 2, 96, 80
    q, k, v, u = 0.1 * rnd(S, H, dk), 0.1 * rnd(S, G, dk, seed=1), rnd(S, G, dv, seed=2), rnd(dk, seed=3)
    u = 5 * u / u.norm()
    q[:], k[far] = u, u
    rule = ScoreRule(log_amount=torch.full((H,), 1.5), log_rate=torch.full((H,), 0.3))
    want, rd = want_attention(q.bfloat16().float(), k.bfloat16().float(), v.bfloat16().float(), 1.0, rule), on_gpu(rule)
    out = torch.empty(1, S, H, dv, dtype=BF16, device="cuda")
    attn_ops.prompt_attention(dev(q, BF16)[None], dev(k, BF16)[None], dev(v, BF16)[None], 1.0, out, rd)
    close(out.view(S, -1), want, 1.5e-2)
    assert torch.allclose(out[0, far:].float().cpu().view(-1, G, H // G, dv), v[far].view(1, G, 1, dv).expand(S - far, G, H // G, dv), atol=0.1)
    (kc, bt), (vc, _) = paged(k, 16, BF16), paged(v, 16, BF16)
    got = paged_ops.paged_attention_decode(dev(q[-1:], BF16).view(1, -1), kc, vc, bt, torch.tensor([S], dtype=torch.int32, device="cuda"), 1.0, rule=rd)
    close(got, want[-1:], 1.5e-2)


# ---- recurrent mixers -------------------------------------------------------------------------------------------------------
SEGS = [(0, 37, 2, 0), (37, 1, 0, 9), (38, 16, 1, 3), (54, 2, 3, 0), (56, 1, 4, 0), (57, 150, 5, 8)]
ROWS = 207


def strided(rows, cols, lead, extra, seed, dtype):
    return dev(rnd(rows, lead + cols + extra, seed=seed).to(dtype))[:, lead:lead + cols]


@BOTH
@pytest.mark.parametrize("aligned", [True, False])
@pytest.mark.parametrize("inner,n", [(256, 24), (130, 16), (96, 5), (64, 4), (72, 8), (40, 64), (36, 100), (24, 256), (33, 17), (5000, 16), (2500, 32), (16, 1), (12, 12), (300, 16)])
def test_selective_scan(inner, n, aligned, dtype):
    extra = 8 if aligned else 1
    x, z, low = (strided(ROWS, c, 8 if aligned else 3, extra, s, dtype) for c, s in ((inner, 0), (inner, 1), (2 * n, 2)))
    dt = strided(ROWS, inner, 4 if aligned else 1, extra, 3, F32)
    A, D, bias = -(rnd(inner, n, seed=4).abs() + 0.01), rnd(inner, seed=5), rnd(inner, seed=6) - 3
    state = 0.3 * rnd(6, inner, (n + 3) // 4 * 4, seed=7)
    state[2:5] = float("nan")                                           # slots of sequences that begin
    sc, y = state.clone(), torch.full((ROWS, inner + 8), 3.0, dtype=dtype, device="cuda")
    want = selective_scan(x.cpu(), dt.cpu(), low[:, :n].cpu(), low[:, n:].cpu(), z.cpu(), A=A, D=D, dt_bias=bias, state=sc, seg=Segments.of(SEGS, "cpu"), scale=0.7).float()
    sd = dev(state)
    selective_scan(x, dt, low[:, :n], low[:, n:], z, A=dev(A), D=dev(D), dt_bias=dev(bias), state=sd, seg=Segments.of(SEGS, "cuda"), scale=0.7, out=y[:, :inner])
    close(y[:, :inner], want, 6e-3 if dtype == BF16 else 5e-6)
    close(sd[:, :, :n], sc[:, :, :n], 1e-5)
    assert bool((y[:, inner:] == 3.0).all())


def test_selective_scan_remembers_far_back():
    """One impulse, decays close to 1: what is left of it after thousands of tokens, in one portion and in pieces."""
    T, inner, n = 4000, 32, 16
    x = torch.zeros(T, inner)
    x[3] = 1.0
    one = torch.ones(T, n)
    dt, A = torch.zeros(T, inner), -torch.logspace(-5, -2.5, inner * n).view(inner, n)
    kw = dict(D=torch.zeros(inner), dt_bias=torch.zeros(inner))
    step = float(torch.log(torch.tensor(2.0)))
    left = step * torch.exp(step * A.double() * (T - 1 - 3)).sum(1).float()
    for cuts in ([T], [2, 4, 5, 1300, 1301, T]):
        for dtype in (BF16, F32):
            st, lo = torch.full((1, inner, n), 1e4, device="cuda"), 0
            for hi in cuts:
                y = selective_scan(*(dev(t[lo:hi], d) for t, d in ((x, dtype), (dt, F32), (one, dtype), (one, dtype), (torch.full((T, inner), 30.0), dtype))), A=dev(A),
                                   state=st, seg=Segments.of([(0, hi - lo, 0, lo)], "cuda"), scale=1 / 30.0, **{k: dev(v) for k, v in kw.items()})
                lo = hi
            close(y[-1], left, 6e-3 if dtype == BF16 else 2e-4, (cuts, dtype))        # rounded decays, 4000 times
            close(st[0].sum(1), left, 4e-4, "state")


@BOTH
@pytest.mark.parametrize("H,n,dv", [(2, 32, 64), (3, 64, 128), (1, 128, 72), (4, 16, 24), (3, 12, 10), (1, 144, 40), (2, 24, 200)])
def test_fixed_decay(H, n, dv, dtype):
    decay = torch.tensor([1.0, 0.9990234375, 0.5, 0.93][:H])
    xbc = strided(ROWS, H * (dv + 2 * n), 0, 8, n, dtype)
    state = 0.3 * rnd(6, H, n, (dv + 3) // 4 * 4, seed=7)
    state[2:5] = 1e4
    sc = state.clone()
    kw = dict(heads=H, groups=H, vdim=dv, n=n)
    want = state_space(xbc.cpu(), decay=decay, state=sc, seg=Segments.of(SEGS, "cpu"), **kw).float()
    sd = dev(state)
    got = state_space(xbc, decay=dev(decay), state=sd, seg=Segments.of(SEGS, "cuda"), **kw)
    close(got, want, 1e-2 if dtype == BF16 else 5e-6)
    close(sd[..., :dv], sc[..., :dv], 2e-5 if dtype == BF16 else 5e-6)


@pytest.mark.parametrize("T,cuts", [(2600, []), (2600, [1, 130, 131, 1500]), (700, [64, 128, 129, 600])])
def test_fixed_decay_over_spans(T, cuts):
    """Long portions are cut into spans that run side by side; a far token still weighs what its decay leaves."""
    H, n, dv = 2, 64, 64
    decay = torch.tensor([0.9990234375, 0.984375])
    v, k, q = (rnd(T, H, s, seed=i).bfloat16().float() for i, s in enumerate((dv, n, n)))
    k[5], q[T - 1] = 12 * k[5], k[5]
    q = q.bfloat16().float()
    k = k.bfloat16().float()
    packed = torch.cat([t.reshape(T, -1) for t in (v, k, q)], 1)
    want = O.retain(q.double(), k.double(), v.double(), decay.double()).float().reshape(T, -1)
    st, out, lo = torch.full((1, H, n, dv), 1e4, device="cuda"), [], 0
    for hi in [*cuts, T]:
        out.append(state_space(dev(packed[lo:hi], BF16), decay=dev(decay), state=st, heads=H, groups=H, vdim=dv, n=n, seg=Segments.of([(0, hi - lo, 0, lo)], "cuda")))
        lo = hi
    got = torch.cat(out).float().cpu()
    rel = (got - want).view(T, H, dv).pow(2).mean(-1).sqrt() / want.view(T, H, dv).pow(2).mean(-1).sqrt()
    assert float(rel.max()) < 2e-2 and float(rel.median()) < 6e-3


@BOTH
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5])
@pytest.mark.parametrize("channels", [40, 37, 1200])
def test_convolution_without_activation(channels, taps, dtype):
    x, w, state = strided(ROWS, channels, 0, 8, 1, dtype), rnd(channels, taps, seed=2), rnd(6, taps - 1, channels, seed=3).to(dtype)
    sc, sd = state.clone(), dev(state)
    want = short_conv(x.cpu(), w, None, sc, Segments.of(SEGS, "cpu"), silu=False).float()
    close(short_conv(x, dev(w), None, sd, Segments.of(SEGS, "cuda"), silu=False), want, 5e-3 if dtype == BF16 else 1e-5)
    assert torch.equal(sd.cpu(), sc)


@BOTH
@pytest.mark.parametrize("parts,m", [(2, 64), (3, 24), (3, 10), (1, 200), (4, 256)])
def test_norm_per_head_without_a_weight(parts, m, dtype):
    y, z = rnd(19, parts * m).to(dtype), rnd(19, parts * m, seed=1).to(dtype)
    want = O.unit_rms(y.float().view(19, parts, m), 1e-3).reshape(19, -1) * O.silu(z.float())
    close(gated_norm(dev(y), dev(z), None, parts, 1e-3, gate_first=False), want, 6e-3 if dtype == BF16 else 1e-5)


# ---- norms, feed-forwards ---------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("n", [24, 90, 192, 1032, 4096])
def test_residual_add_with_a_norm_behind(n, dtype):
    T, g = 19, torch.tensor(0.7)
    x, y = rnd(T, n), rnd(T, n, seed=1)
    gd, tol, xd, h = torch.full((n,), 0.7, device="cuda"), 5e-3 if dtype == BF16 else 1e-5, dev(x.clone()), torch.empty(T, n, dtype=dtype, device="cuda")
    residual_norm(dev(y), None, None, 1e-3, True, x=xd, h=h, next_gamma=gd)
    assert torch.equal(xd.cpu(), x + y)                                  # a 32-bit sum
    close(h, O.scalar_norm(x + y, g, 1e-3), tol)
    xd = dev(x.clone())
    residual_norm(dev(y), None, None, 1e-3, True, x=xd)
    assert torch.equal(xd.cpu(), x + y)
    rows, slots = rnd(60, n, seed=4).to(dtype), torch.randint(0, 60, (T, 3), generator=torch.Generator().manual_seed(1))
    want = x + rows.float()[slots].sum(1)
    xd = dev(x.clone())
    residual_norm(dev(rows), None, None, 1e-3, True, x=xd, h=h, next_gamma=gd, routed=(dev(slots.reshape(-1).to(torch.int32)), None))
    close(xd, want, 1e-6)
    close(h, O.scalar_norm(want, g, 1e-3), tol)


@BOTH
@pytest.mark.parametrize("T,E,k,ff", [(40, 8, 2, 64), (9, 5, 5, 24), (300, 16, 1, 40), (3, 1, 1, 16), (33, 12, 4, 20)])
def test_expert_weights_multiply_the_input(T, E, k, ff, dtype):
    d, f8 = 48, (ff + 7) // 8 * 8
    x, router = rnd(T, d).to(dtype), 2 * rnd(E, d, seed=1)
    w = {f"e{e}.{n}": (rnd(*s, seed=10 * e + i) * s[1] ** -0.5).to(dtype) for e in range(E) for i, (n, s) in enumerate((("gate", (ff, d)), ("up", (ff, d)), ("down", (d, ff))))}
    wf = {**{n: t.float() for n, t in w.items()}, "router": router}
    want = O.routed_ff(x.float(), wf, "", {"router": {"top": k}})
    idx, ws = moe_ops.route_sigmoid(dev(x.float() @ router.T), k)
    pl = moe_ops.plan(idx, E)
    w1, w2 = torch.zeros(E, 2 * f8, d, dtype=dtype), torch.zeros(E, d, f8, dtype=dtype)
    for e in range(E):
        w1[e, :ff], w1[e, f8:f8 + ff], w2[e, :, :ff] = w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"]
    gu = moe_ops.grouped_gemm(moe_ops.scatter_tokens(dev(x), pl), dev(w1), pl)
    y = moe_ops.grouped_gemm(moe_ops.swiglu_rows(gu, pl, weights=ws), dev(w2), pl)
    close(y[pl.slot_pos.long()].float().view(T, k, d).sum(1), want, 1.5e-2 if dtype == BF16 else 1e-5)


# ---- the whole model ---------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_prefill_portions_and_decoding_agree_with_the_plain_model(name, dtype):
    C.check_prefill_portions_and_decode(name, "cuda", dtype)


@BOTH
def test_long_prompt_in_portions(dtype):
    """A prompt of several tiles, chunks and slices of the kernels, cut at and around their edges."""
    C.check_prefill_portions_and_decode("dense", "cuda", dtype, 700, {"whole": [], "around tiles": [63, 64, 66, 128, 129, 191, 256, 320, 511, 513], "halves": [350],
                                                                     "two and then the rest": [2, 4, 600, 602]})


@BOTH
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_mixed_batches_with_reused_pages(name, dtype):
    C.check_mixed_batch_with_reused_pages(name, "cuda", dtype)


@BOTH
@pytest.mark.parametrize("name", ["varied", "dense"])
def test_long_decoding(name, dtype):
    C.check_long_decoding(name, "cuda", dtype, 330 if name == "dense" else 110)


def test_first_tokens_of_a_sequence():
    for name in ("varied", "wide"):
        cfg = C.CONFIGS[name]
        w = C.weights(cfg, 8)
        for n in (1, 2, 3):
            r = C.runner(cfg, w, "cuda")
            C.poison(r)
            toks = C.tokens(cfg, n, n)
            C.assert_logits(C.feed(r, 0, toks, []), C.reference(cfg, w, toks), F32, (name, n))


def test_greedy_generation_through_the_engine_in_32_bit():
    cfg = C.CONFIGS["wide"]
    w = C.weights(cfg, 6)
    r = C.runner(cfg, w, "cuda", F32, blocks=60)
    C.poison(r)
    eng = ServingEngine(r, max_batch_size=3, prefill_chunk=64)
    prompts = [C.tokens(cfg, n, 20 + n) for n in (5, 170, 33, 1)]
    ids = [eng.submit(p, 8) for p in prompts]
    eng.run_to_completion()
    wd = {k: v.double() for k, v in w.items()}
    for p, rid in zip(prompts, ids):
        assert eng.scheduler.get(rid).generated == O.greedy(cfg, wd, p, 8)
    assert r.cache.free_blocks == 60


def test_generation_in_bf16_does_not_depend_on_the_batch():
    """The same request alone and beside others, whole and in portions: logits agree beyond rounding, so greedy tokens do."""
    cfg = C.CONFIGS["wide"]
    w = C.weights(cfg, 6)
    prompts = [C.sequence(cfg, w, n, 50 + n, BF16) for n in (60, 7, 90)]
    alone = [ServingEngine(C.runner(cfg, w, "cuda", BF16, blocks=60)).generate(p, 4) for p in prompts]
    eng = ServingEngine(C.runner(cfg, w, "cuda", BF16, blocks=60), max_batch_size=4, prefill_chunk=50)
    ids = [eng.submit(p, 4) for p in prompts]
    eng.run_to_completion()
    same = sum(eng.scheduler.get(r).generated[0] == a[0] for r, a in zip(ids, alone))
    assert same >= 2
