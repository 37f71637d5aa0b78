"""Looped decoders (Bikilix) on the GPU: every kernel against plain math, then the step function, the cache and the engine against
tests/looped_oracle.py in bf16 and in true 32-bit."""
import pytest
import torch

import looped_checks as C
import looped_oracle as O
from rustral_b200.models.layered import RotarySpec
from rustral_b200.ops import (ScoreRule, embedding_residual, gemm, head_prep_, head_product, latent_decode, latent_prep_, residual_norm, rotary_table,
                              rotate_pairs_)
from rustral_b200.ops import attention as attn_ops
from rustral_b200.ops import latent as latent_ops
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
    spec = RotarySpec.from_json(rot)
    return rotary_table(pos.cuda(), torch.tensor(spec.frequencies(), dtype=torch.float64, device="cuda"), spec.magnitude)


def turned(x3, pos, rot):
    return O.rotate(x3.double(), pos, rot).float()


# ---- positions ---------------------------------------------------------------------------------------------------------
def test_rotary_table_far_out():
    rot = dict(dims=40, base=1e5, scaling=dict(factor=6.0, original=700, fast=16.0, slow=1.0))
    pos = torch.tensor([0, 1, 17, 4095, 131071, 10 ** 6])
    spec = RotarySpec.from_json(rot)
    a = pos.double()[:, None] * torch.tensor(spec.frequencies(), dtype=torch.float64)
    want = torch.stack([torch.cos(a), torch.sin(a)], -1) * spec.magnitude
    assert float((table_of(rot, pos).cpu().double() - want).abs().max()) < 1e-6


@BOTH
@pytest.mark.parametrize("heads,pitch,first,dims", [(3, 48, 16, 32), (1, 24, 8, 16), (5, 20, 6, 14), (2, 10, 0, 2), (4, 64, 0, 64), (2, 40, 8, 24)])
def test_rotate_pairs(heads, pitch, first, dims, dtype):
    rot, pos = dict(dims=dims, base=700.0), torch.tensor([0, 5, 90, 3, 3, 1000, 7])
    x = rnd(7, heads * pitch + 8).to(dtype)
    want = x.float().clone()
    v = want[:, :heads * pitch].reshape(7, heads, pitch)
    v[..., first:] = turned(v[..., first:], pos, rot)
    want[:, :heads * pitch] = v.reshape(7, -1)
    xd = dev(x)
    rotate_pairs_(xd, heads, pitch, first, table_of(rot, pos))
    close(xd, want, 5e-3 if dtype == BF16 else 1e-5)
    assert torch.equal(xd[:, heads * pitch:].cpu(), x[:, heads * pitch:])


@BOTH
@pytest.mark.parametrize("normed", [False, True])
@pytest.mark.parametrize("H,G,dk,dv,dims", [(4, 2, 64, 64, 32), (6, 2, 104, 40, 28), (2, 2, 128, 128, 128), (4, 1, 24, 16, 2), (3, 3, 20, 12, 6), (2, 1, 40, 8, 20),
                                            (1, 1, 13, 7, 12), (4, 2, 200, 64, 64)])
def test_head_prep_with_positions(H, G, dk, dv, dims, normed, dtype):
    T = 9
    rot, pos = dict(dims=dims, base=900.0), torch.arange(T) * 37
    p = rnd(T, H * dk + G * (dk + dv) + 8, seed=dk).to(dtype)
    gq, gk = (rnd(dk, seed=1).to(dtype), rnd(dk, seed=2).to(dtype)) if normed else (None, None)
    slots = torch.tensor([11, 0, 3, -1, 5, 6, 7, 8, 1])
    q, k = p[:, :H * dk].float().reshape(T, H, dk), p[:, H * dk:(H + G) * dk].float().reshape(T, G, dk)
    if normed:
        q, k = O.rms_norm(q, gq.float(), 1e-3), O.rms_norm(k, gk.float(), 1e-3)
    want_q, want_k = turned(q, pos, rot), turned(k, pos, rot)
    kc, vc, pd = torch.zeros(3, 4, G, dk, dtype=dtype, device="cuda"), torch.zeros(3, 4, G, dv, dtype=dtype, device="cuda"), dev(p)
    head_prep_(pd, H, G, dk, dv, q_gamma=None if gq is None else dev(gq), k_gamma=None if gk is None else dev(gk), eps=1e-3, k_cache=kc, v_cache=vc,
               slots=dev(slots), rot=table_of(rot, pos))
    tol = 6e-3 if dtype == BF16 else 1e-5
    close(pd[:, :H * dk].view(T, H, dk), want_q, tol)
    keep = slots >= 0
    close(kc.view(12, G, dk)[dev(slots[keep])], want_k[keep], tol)
    ov = (H + G) * dk
    assert torch.equal(vc.view(12, G * dv)[dev(slots[keep])].cpu(), p[keep][:, ov:ov + G * dv]) and torch.equal(pd[:, ov:].cpu(), p[:, ov:])
    assert float(kc.view(12, -1)[[2, 4, 9, 10]].abs().max()) == 0


@BOTH
@pytest.mark.parametrize("q_rank,R,dr,dims", [(72, 56, 24, 24), (1536, 512, 64, 64), (40, 136, 16, 8), (7, 9, 4, 4), (2000, 24, 6, 6), (8, 8, 2, 2)])
def test_latent_prep(q_rank, R, dr, dims, dtype):
    T, oq = 9, 8
    ok = oq + (q_rank + 7) // 8 * 8
    rot, pos = dict(dims=dims, base=900.0), torch.arange(T) * 211
    p, gq, gk = rnd(T, ok + (R + dr + 7) // 8 * 8 + 16, seed=R).to(dtype), rnd(q_rank, seed=1), rnd(R, seed=2)
    slots = torch.tensor([11, 0, 3, -1, 5, 6, 7, 8, 1])
    want = p.float().clone()
    want[:, oq:oq + q_rank] = O.rms_norm(want[:, oq:oq + q_rank], gq, 1e-3)
    want[:, ok:ok + R] = O.rms_norm(want[:, ok:ok + R], gk, 1e-3)
    want[:, ok + R:ok + R + dr] = turned(want[:, None, ok + R:ok + R + dr], pos, rot)[:, 0]
    cache, pd = torch.zeros(3, 4, 1, R + dr, dtype=dtype, device="cuda"), dev(p)
    latent_prep_(pd, oq, q_rank, ok, R, dr, q_gamma=dev(gq), kv_gamma=dev(gk), eps=1e-3, table=table_of(rot, pos), cache=cache, slots=dev(slots))
    close(pd, want, 6e-3 if dtype == BF16 else 1e-5)
    keep = slots >= 0
    assert torch.equal(cache.view(12, -1)[dev(slots[keep])], pd[dev(keep)][:, ok:ok + R + dr]) and float(cache.view(12, -1)[[2, 4, 9, 10]].abs().max()) == 0


# ---- latent attention ------------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("rows", [1, 5, 64, 130])
@pytest.mark.parametrize("heads,n,k,tail,dims", [(3, 72, 40, 24, 24), (3, 512, 128, 64, 64), (16, 128, 512, 0, 0), (2, 40, 24, 8, 4), (5, 20, 12, 6, 6), (1, 8, 8, 0, 0),
                                                 (20, 136, 128, 64, 64)])
def test_head_product(heads, n, k, tail, dims, rows, dtype):
    x_head = k + tail
    x = rnd(rows, heads * x_head + 8, seed=rows).to(dtype)[:, :heads * x_head]
    w = (rnd(heads * n, k, seed=1) * k ** -0.5).to(dtype)
    rot, pos = dict(dims=dims, base=100.0), torch.arange(rows) * 3
    table = table_of(rot, pos) if tail else None
    x3 = x.float().reshape(rows, heads, x_head)
    plain = torch.einsum("thk,hnk->thn", x3[..., :k], w.float().view(heads, n, k))
    wt = w.view(heads, n, k).transpose(1, 2).contiguous().view(heads * k, n)
    gate = rnd(rows, heads * n + 8, seed=4).to(dtype)[:, 8:]
    for transposed, ww in ((False, w), (True, wt)):
        for g in (None, gate):
            want = plain if g is None else plain * O.sigmoid(g.float()).reshape(rows, heads, n)
            if tail:
                want = torch.cat([want, turned(x3[..., k:], pos, rot)], -1)
            buf = torch.full((rows, heads * (n + tail) + 8), 3.0, dtype=dtype, device="cuda")
            gd = None if g is None else dev(torch.cat([g[:, :8], g], 1))[:, 8:]
            head_product(dev(x), x_head, dev(ww), heads, n, k, transposed=transposed, gate=gd, tail=tail, table=table, out=buf[:, :heads * (n + tail)])
            close(buf[:, :heads * (n + tail)], want.reshape(rows, -1), 1e-2 if dtype == BF16 else 1e-5, (transposed, g is not None))
            assert bool((buf[:, heads * (n + tail):] == 3.0).all())


def paged_slots(slots, bs, dtype, seed=0):
    """One sequence's slots on scattered pages among pages full of other values."""
    S, W = slots.shape
    n = -(-S // bs)
    perm = torch.randperm(n + 5, generator=torch.Generator().manual_seed(seed))[:n]
    c = torch.full((n + 5, bs, 1, W), 1e4)
    for j in range(S):
        c[perm[j // bs], j % bs, 0] = slots[j]
    return c.to(dtype), perm.to(torch.int32)


LATENT = [  # context, heads, rank, rotated, page
    (1, 5, 80, 24, 16), (64, 5, 80, 24, 16), (65, 5, 80, 24, 16), (128, 16, 128, 64, 16), (129, 17, 128, 64, 16), (500, 40, 512, 64, 16), (700, 16, 512, 64, 64),
    (257, 3, 256, 128, 4), (300, 33, 264, 8, 16), (90, 5, 72, 16, 16), (400, 2, 8, 8, 1), (200, 8, 512, 128, 16), (63, 1, 16, 64, 16), (150, 20, 136, 64, 16),
]


def latent_want(q, slots, R, scale):
    return (O.softmax_rows(q.double() @ slots.double().T * scale) @ slots.double()[:, :R]).float()


@pytest.mark.parametrize("case", LATENT, ids=str)
@pytest.mark.parametrize("width", [0, 400])
def test_latent_decode(case, width):
    ctx, H, R, dr, bs = case
    scale, W = 1.5 * (R + dr) ** -0.5, R + dr
    lens = [ctx, 1 + ctx // 3, max(1, ctx - 1)]                      # unequal sequences in one batch
    qs = [rnd(H, W, seed=n).bfloat16().float() for n in lens]
    sl = [rnd(n, W, seed=n + 1).bfloat16().float() for n in lens]
    want = torch.stack([latent_want(q, s, R, scale).reshape(-1) for q, s in zip(qs, sl)])
    for dtype in (BF16, F32):
        pages = [paged_slots(s, bs, dtype, i) for i, s in enumerate(sl)]
        bt = torch.zeros(3, max(len(t) for _, t in pages) + 3 + width // bs, dtype=torch.int32)   # a wide table: most slices are empty
        at = 0
        for i, (c, t) in enumerate(pages):
            bt[i, :len(t)] = t + at
            at += c.shape[0]
        cache, bt = dev(torch.cat([c for c, _ in pages])), dev(bt)
        q = dev(torch.stack(qs).view(3, -1), dtype)
        rows = paged_ops.paged_attention_rows(q, cache, cache[..., :R], bt, torch.arange(3, dtype=torch.int32, device="cuda"),
                                              torch.tensor(lens, device="cuda") - 1, scale)
        close(rows, want, 1e-2 if dtype == BF16 else 1e-5, "rows")
        if dtype == BF16:
            assert latent_ops.latent_decode_supported(q, R, dr)
            close(latent_decode(q, cache, R, bt, torch.tensor(lens, dtype=torch.int32, device="cuda"), scale), want, 1e-2, "decode")


@pytest.mark.parametrize("batch", [1, 16, 64])
def test_latent_decode_slices_by_batch(batch):
    """Slices get shorter for small batches; the result does not depend on it."""
    H, R, dr, n = 3, 80, 24, 600
    s, q = rnd(n, R + dr, seed=5).bfloat16().float(), rnd(H, R + dr, seed=6).bfloat16().float()
    cache, t = paged_slots(s, 16, BF16)
    bt = dev(t)[None].expand(batch, -1).contiguous()
    ctx = torch.tensor([n - i for i in range(batch)], dtype=torch.int32)
    got = latent_decode(dev(q.view(1, -1), BF16).expand(batch, -1).contiguous(), dev(cache), R, bt, dev(ctx), 0.1)
    close(got, torch.stack([latent_want(q, s[:n - i], R, 0.1).reshape(-1) for i in range(batch)]), 1e-2)


@pytest.mark.parametrize("ctx,far", [(700, 0), (700, 15), (700, 16), (700, 63), (700, 64), (700, 127), (700, 128), (700, 511), (700, 512), (700, 699), (700, 698), (129, 128)])
def test_latent_decode_finds_one_key_that_stands_out(ctx, far):
    H, R, dr = 5, 128, 64
    s, q = 0.3 * rnd(ctx, R + dr, seed=1), 0.3 * rnd(H, R + dr, seed=2)
    u = rnd(R + dr, seed=3)
    u = u / u.norm()
    q[3], s[far] = 7 * u, 7 * u
    s, q = s.bfloat16().float(), q.bfloat16().float()
    cache, t = paged_slots(s, 16, BF16)
    got = latent_decode(dev(q.view(1, -1), BF16), dev(cache), R, dev(t)[None].contiguous(), torch.tensor([ctx], dtype=torch.int32, device="cuda"), 1.0)
    close(got.view(H, R)[3], s[far, :R], 2e-2)


@pytest.mark.parametrize("ctx", [1, 17, 63, 64, 65, 130, 1000])
@pytest.mark.parametrize("R,dr,bs", [(80, 24, 16), (512, 64, 16), (256, 32, 64), (128, 64, 4)])
def test_latent_decode_does_not_read_what_a_page_held_before(ctx, R, dr, bs):
    """Rows of the last page behind the context can hold anything, also what is not a number."""
    H = 18
    s, q = rnd(ctx, R + dr, seed=1).bfloat16().float(), rnd(H, R + dr, seed=2).bfloat16().float()
    cache, t = paged_slots(s, bs, BF16)
    used = torch.zeros(cache.shape[:2], dtype=torch.bool)
    for j in range(ctx):
        used[t[j // bs], j % bs] = True
    cache[~used] = float("nan")
    bt = torch.cat([t, torch.zeros(9, dtype=torch.int32)])[None]
    got = latent_decode(dev(q.view(1, -1), BF16), dev(cache), R, dev(bt), torch.tensor([ctx], dtype=torch.int32, device="cuda"), 0.1)
    close(got.view(H, R), latent_want(q, s, R, 0.1), 1e-2)


def test_row_kernel_with_more_value_columns_than_one_block():
    R, dr, H = 1100, 16, 2
    s, q = rnd(40, R + dr).bfloat16().float(), rnd(H, R + dr, seed=1).bfloat16().float()
    for dtype in (BF16, F32):
        cache, t = paged_slots(s, 16, dtype)
        cache = dev(cache)
        got = paged_ops.paged_attention_rows(dev(q.view(1, -1), dtype), cache, cache[..., :R], dev(t)[None].contiguous(),
                                             torch.zeros(1, dtype=torch.int32, device="cuda"), torch.tensor([39], device="cuda"), 0.05)
        close(got.view(H, R), latent_want(q, s, R, 0.05), 1e-2 if dtype == BF16 else 1e-5)


SPLIT = [  # rows, keys, heads, unrotated, rotated, value size
    (1, 1, 2, 64, 64, 64), (2, 2, 2, 8, 8, 8), (130, 130, 3, 40, 24, 48), (300, 300, 3, 128, 64, 128), (257, 700, 2, 128, 64, 128), (513, 513, 2, 128, 64, 64),
    (2, 400, 4, 128, 64, 128), (140, 141, 2, 24, 16, 72), (600, 1000, 2, 72, 40, 24), (384, 1024, 1, 64, 48, 104), (129, 900, 6, 64, 32, 128), (700, 900, 2, 40, 8, 96),
    (1, 640, 20, 128, 64, 128), (1200, 1200, 1, 128, 64, 128),
]


@pytest.mark.parametrize("case", SPLIT, ids=str)
def test_flash_kernel_with_a_shared_key_part(case):
    L, S, H, dn, dr, dv = case
    r = lambda *s, seed: rnd(*s, seed=seed).bfloat16().float()
    q, k, kr, v, gate = 1.5 * r(L, H, dn + dr, seed=1), r(S, H, dn, seed=2), r(S, dr, seed=3), r(S, H, dv, seed=4), r(L, H * dv, seed=5)
    q = q.bfloat16().float()
    scale = 1.3 * (dn + dr) ** -0.5
    full = torch.zeros(S, H, dn + dr)
    full[S - L:] = q
    want = O.attend(full.double(), torch.cat([k, kr[:, None].expand(S, H, dr)], -1).double(), v.double(), scale)[S - L:].float().reshape(L, -1)
    both = dev(torch.cat([k.reshape(S, -1), v.reshape(S, -1)], 1), BF16)                 # keys of all heads beside values of all heads
    wide = torch.full((S, dr + 24), 9.0, dtype=BF16, device="cuda")
    wide[:, 16:16 + dr] = dev(kr, BF16)
    krd, qd = wide[:, 16:16 + dr], dev(q, BF16)
    assert attn_ops.split_supported(dn, dr, dv, qd.view(L, -1), both, krd)
    for g in (None, gate):
        out = torch.full((1, L, H, dv), 7.0, dtype=BF16, device="cuda")
        attn_ops.prompt_attention_split(qd[None], both[:, :H * dn].view(1, S, H, dn), both[:, H * dn:].view(1, S, H, dv), krd, scale, out,
                                        gate=None if g is None else dev(g, BF16))
        close(out.view(L, -1), want if g is None else want * O.sigmoid(g), 1.5e-2, g is not None)


@pytest.mark.parametrize("far", [0, 127, 128, 255, 256, 300, 511, 512])
@pytest.mark.parametrize("part", ["unrotated", "rotated"])
def test_flash_kernel_finds_one_key_that_stands_out(far, part):
    """By either part of the key, wherever it is; no row before it sees it."""
    S, H, dn, dr, dv = 640, 2, 128, 64, 64
    q, k, kr, v = 0.2 * rnd(S, H, dn + dr), 0.2 * rnd(S, H, dn, seed=1), 0.2 * rnd(S, dr, seed=2), rnd(S, H, dv, seed=3)
    lo, n = (0, dn) if part == "unrotated" else (dn, dr)
    u = rnd(n, seed=4)
    u = 6 * u / u.norm()
    q[:, :, lo:lo + n] = u
    if part == "unrotated":
        k[far] = u
    else:
        kr[far] = u
    out = torch.empty(1, S, H, dv, dtype=BF16, device="cuda")
    attn_ops.prompt_attention_split(dev(q, BF16)[None], dev(k, BF16)[None], dev(v, BF16)[None], dev(kr, BF16), 1.0, out)
    o = out[0].float().cpu()
    assert torch.allclose(o[far:], v[far].bfloat16().float().expand(S - far, H, dv), atol=0.03)
    if far:
        assert float((o[far - 1] - v[far]).abs().max()) > 0.3


WINDOWS = [  # rows, keys, heads, kv heads, dk, dv, window
    (1, 1, 2, 1, 64, 64, 8), (130, 130, 6, 2, 88, 88, 140), (300, 300, 4, 1, 88, 56, 48), (257, 700, 2, 1, 128, 128, 300), (513, 513, 2, 1, 128, 64, 129),
    (2, 200, 4, 2, 48, 40, 63), (140, 141, 2, 1, 32, 72, 1), (600, 1000, 2, 2, 64, 64, 500), (700, 900, 2, 1, 80, 96, 37), (129, 900, 6, 3, 64, 32, 4096),
]


@pytest.mark.parametrize("case", WINDOWS, ids=str)
def test_flash_kernel_with_a_plain_window(case):
    L, S, H, G, dk, dv, window = case
    r = lambda *s, seed: rnd(*s, seed=seed).bfloat16().float()
    q, k, v = (2 * r(L, H, dk, seed=1)).bfloat16().float(), r(S, G, dk, seed=2), r(S, G, dv, seed=3)
    rule, scale = ScoreRule(window=window), 1.3 * dk ** -0.5
    full = torch.zeros(S, H, dk)
    full[S - L:] = q
    want = O.attend(full.double(), k.double(), v.double(), scale, window)[S - L:].float().reshape(L, -1)
    for first in {0, rule.key_ranges(S - L)[1]}:                       # all keys, and those that the portion gathers
        out = torch.full((1, L, H, dv), 7.0, dtype=BF16, device="cuda")
        attn_ops.prompt_attention(dev(q, BF16)[None], dev(k[first:], BF16)[None], dev(v[first:], BF16)[None], scale, out, rule)
        close(out.view(L, -1), want, 1.5e-2, first)


# ---- norms, feed-forwards, products ---------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("n", [24, 90, 192, 1032, 4096])
def test_norm_behind_and_norm_in_front(n, dtype):
    T = 19
    x, y, w, nxt = rnd(T, n), rnd(T, n, seed=1), 0.3 * rnd(n, seed=2), 0.3 * rnd(n, seed=3)
    want = x + O.centred_norm(y, w, 1e-3)
    wd, nd = dev(1 + w), dev(1 + nxt)
    tol = 5e-3 if dtype == BF16 else 1e-5
    xd, h = dev(x.clone()), torch.empty(T, n, dtype=dtype, device="cuda")
    residual_norm(dev(y), wd, None, 1e-3, True, x=xd, h=h, next_gamma=nd)
    close(xd, want, 1e-5)                                              # the residual is 32-bit in both
    close(h, O.centred_norm(want, nxt, 1e-3), tol)
    pair, xd = torch.full((T, 2 * n), 3.0, dtype=dtype, device="cuda"), dev(x.clone())
    residual_norm(dev(y), wd, None, 1e-3, True, x=xd, h=pair[:, :n])
    assert torch.equal(pair[:, :n].float(), xd.to(dtype).float()) and bool((pair[:, n:] == 3.0).all())
    close(residual_norm(dev(want), nd, None, 1e-3, True, h=torch.empty(T, n, dtype=dtype, device="cuda")), O.centred_norm(want, nxt, 1e-3), tol)
    rows, slots, ws = rnd(60, n, seed=4).to(dtype), torch.randint(0, 60, (T, 3), generator=torch.Generator().manual_seed(1)), torch.rand(T, 3)
    want = x + O.centred_norm((rows.float()[slots] * ws[..., None]).sum(1), w, 1e-3)
    xd = dev(x.clone())
    residual_norm(dev(rows), wd, None, 1e-3, True, x=xd, h=h, next_gamma=nd, routed=(dev(slots.reshape(-1).to(torch.int32)), dev(ws)))
    close(xd, want, 1e-5)
    close(h, O.centred_norm(want, nxt, 1e-3), tol)


@pytest.mark.parametrize("T,E,k,groups,keep,best", [(40, 8, 2, 4, 2, 2), (9, 12, 3, 3, 1, 2), (33, 6, 1, 6, 1, 2), (70, 9, 4, 3, 2, 1), (5, 10, 10, 1, 1, 2), (3, 1, 1, 1, 1, 2),
                                                    (300, 64, 6, 8, 4, 2), (50, 96, 8, 4, 3, 2), (20, 256, 8, 8, 4, 2), (20, 1000, 40, 10, 5, 2)])
def test_sigmoid_router(T, E, k, groups, keep, best):
    z, corr = 2 * rnd(T, E), 0.7 * rnd(E, seed=1) - 0.5
    for c in (corr, None):
        for renorm in (False, True):
            want_i, want_w = moe_ops.route_sigmoid(z, k, groups, keep, c, best, renorm)
            idx, w = moe_ops.route_sigmoid(dev(z), k, groups, keep, None if c is None else dev(c), best, renorm)
            assert torch.equal(idx.cpu(), want_i)
            close(w, want_w, 1e-5)
    for t in range(min(T, 20) if best == 2 else 0):
        want_i, want_w = O.choose(z[t], corr, k, groups, keep)
        assert moe_ops.route_sigmoid(dev(z[t:t + 1]), k, groups, keep, dev(corr), best)[0][0].tolist() == want_i


def test_router_with_negative_choice_scores():
    z, corr = torch.zeros(1, 6, device="cuda"), torch.tensor([-3.0, -4.0, -0.1, -9.0, -2.0, -2.5], device="cuda")
    idx, w = moe_ops.route_sigmoid(z, 2, 3, 1, corr, 2)
    assert idx.tolist() == [[4, 5]] and w.tolist() == [[0.5, 0.5]]
    assert moe_ops.route_sigmoid(z, 2, 3, 1, corr, 1)[0].tolist() == [[2, 3]] and moe_ops.route_sigmoid(z, 2, 1, 1, corr, 2)[0].tolist() == [[2, 4]]


@BOTH
@pytest.mark.parametrize("F", [16, 88, 50])
def test_clamped_gate(F, dtype):
    gu = (4 * rnd(37, 2 * F)).to(dtype)
    for lim in (0.5, 1.0, 7.0):
        g, u = torch.clamp(gu[:, :F].float(), max=lim), torch.clamp(gu[:, F:].float(), -lim, lim)
        close(moe_ops.swiglu_rows(dev(gu), act="clamped", limit=lim), g * O.sigmoid(1.702 * g) * (u + 1), 5e-3 if dtype == BF16 else 1e-6)


@pytest.mark.parametrize("M,N,K", [(1, 64, 64), (70, 96, 128), (300, 200, 72), (5, 50, 40), (257, 1024, 512)])
def test_product_with_bias_and_squared_relu(M, N, K):
    a, b, bias = rnd(M, K), rnd(N, K, seed=1) * K ** -0.5, rnd(N, seed=2)
    ab, bb, biasb = a.bfloat16(), b.bfloat16(), bias.bfloat16()
    want = torch.relu(ab.float() @ bb.float().T + biasb.float()) ** 2
    close(gemm(dev(ab), dev(bb), bias=dev(biasb), act="relu2"), want, 5e-3)
    close(gemm(dev(ab), dev(bb), bias=dev(biasb), out_dtype=F32), ab.float() @ bb.float().T + biasb.float(), 1e-4)
    close(gemm(dev(ab), dev(bb), act="relu2", out_dtype=F32), torch.relu(ab.float() @ bb.float().T) ** 2, 1e-4)
    want = (a.double() @ b.double().T + bias.double()).float()
    close(gemm(dev(a), dev(b), bias=dev(bias)), want, 1e-5)
    close(gemm(dev(a), dev(b), bias=dev(bias), act="relu2"), torch.relu(want) ** 2, 1e-5)


@BOTH
def test_embedding_beside_the_stream(dtype):
    t = rnd(50, 24).to(dtype)
    pair, ids = torch.zeros(3, 48, dtype=dtype, device="cuda"), torch.tensor([3, 49, 0])
    x, h = embedding_residual(dev(ids), dev(t), 2.5, h=pair[:, 24:])
    assert torch.equal(x.cpu(), t[ids].float() * 2.5) and torch.equal(pair[:, 24:].cpu(), (t[ids].float() * 2.5).to(dtype)) and float(pair[:, :24].abs().max()) == 0


# ---- the whole model ---------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_prefill_portions_and_decoding_agree_with_the_plain_model(name, dtype):
    C.check_prefill_portions_and_decode(name, "cuda", dtype)


@BOTH
def test_long_prompt_in_portions(dtype):
    """A prompt of several windows, tiles and slices of the kernels, cut at and around their edges."""
    C.check_prefill_portions_and_decode("wide", "cuda", dtype, 400, {"whole": [], "around tiles": [63, 64, 66, 128, 129, 191, 256, 320], "halves": [200],
                                                                     "window edges": [69, 70, 71, 149, 150, 151, 153, 299, 301]})


@BOTH
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_mixed_batches_with_reused_pages(name, dtype):
    C.check_mixed_batch_with_reused_pages(name, "cuda", dtype)


@BOTH
@pytest.mark.parametrize("name", ["varied", "wide"])
def test_long_decoding(name, dtype):
    C.check_long_decoding(name, "cuda", dtype, 330 if name == "wide" else 200)


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
    w = C.weights(cfg, 6, BF16)
    prompts = [C.tokens(cfg, n, 50 + n) for n in (60, 7, 161)]
    alone = [ServingEngine(C.runner(cfg, w, "cuda", BF16, blocks=60)).generate(p, 4) for p in prompts]
    eng = ServingEngine(C.runner(cfg, w, "cuda", BF16, blocks=60), max_batch_size=4, prefill_chunk=50)
    ids = [eng.submit(p, 4) for p in prompts]
    eng.run_to_completion()
    same = sum(eng.scheduler.get(r).generated[0] == a[0] for r, a in zip(ids, alone))
    assert same >= 2
