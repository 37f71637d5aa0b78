"""Serving throughput of the pre-norm decoder (Seredra) beside the hybrid one (Vafodra) at equal size, and its kernels beside the like
kernels of the other models against the measured roofline.

    python bench.py --decoders seredra                 # all sizes, JSON line
    python bench.py --decoders seredra --decoder-size medium

Both models have random weights, the same width, attention heads, head size, vocabulary and number of layers, and the same number of
weights that a token passes through (Vafodra's feed-forwards take what its mixers leave).  Timing as in bench.decoders.  Like kernels:
the layered decoder's (Dolurax) for capped attention and head norms, Vafodra's for recurrent mixers and convolutions, the looped one's
(Bikilix) for routing and norms.  The roofline of the selective scan counts its exponentials too (16 a clock and SM).
"""
from __future__ import annotations

import torch

from ..models.layered import LayeredConfig, RotarySpec, hybrid_layers, prenorm_layers
from ..ops import attention as attn_ops
from ..ops import moe as moe_ops
from ..ops import norm as norm_ops
from ..ops import paged as paged_ops
from ..ops import recurrent as rc
from ..ops import rotary as rope_ops
from ..ops.attention import ScoreRule, distance_slopes
from ..ops.heads import head_prep_, row_prep_
from ..ops.matmul import gemm
from .decoders import _peaks, _time, throughput

ORDER, KV_FROM, DENSE = "prapra", {5: 2}, (0, 2, 4)
EXPONENTIALS = 148 * 16 * 1.9e9                # a second, on the special-function units
SIZES = {
    "small": dict(d=2048, vocab=32768, H=16, G=4, dk=128, conv=4, right=dict(inner=4096, state=16, dt_rank=128, conv=4),
                  ret=dict(heads=16, dim=128, vdim=256), ff=8192, E=32, top=4, ffe=1408),
    "medium": dict(d=4096, vocab=65536, H=32, G=8, dk=128, conv=4, right=dict(inner=8192, state=16, dt_rank=256, conv=4),
                   ret=dict(heads=32, dim=128, vdim=256), ff=14336, E=32, top=5, ffe=1920),
    "head64": dict(d=2048, vocab=32768, H=32, G=8, dk=64, conv=4, right=dict(inner=4096, state=32, dt_rank=128, conv=4),
                   ret=dict(heads=32, dim=64, vdim=128), ff=8192, E=64, top=8, ffe=704),
}


def _decays(n: int) -> tuple:
    return tuple(1.0 - 2.0 ** (-5.0 - 7.0 * i / n) for i in range(n))


def _seredra(s) -> LayeredConfig:
    scale = s["dk"] ** -0.5
    heads = dict(heads=s["H"], kv_heads=s["G"], dim=s["dk"], vdim=s["dk"], scale=scale)
    yarn = dict(base=500000.0, factor=8.0, original=4096, fast=32.0, slow=1.0, scaled=True)
    return LayeredConfig(vocab_size=s["vocab"], d_model=s["d"], arch="Seredra", seq_len=16384, layers=prenorm_layers(
        ORDER, dict(heads, conv=s["conv"], temp_coef=0.1, temp_every=4096), dict(heads, softcap=30.0, rot=dict(dims=s["dk"], **yarn)), s["right"],
        (1.0, 1.0), dict(s["ret"], decay=_decays(s["ret"]["heads"]), rot=dict(dims=s["ret"]["dim"], base=10000.0)), s["ff"],
        dict(ff=s["ffe"], experts=s["E"], top=s["top"]), DENSE, KV_FROM))


def _passed(cfg) -> int:
    """Weights of the layers that a token passes through."""
    n = 0
    for s in cfg.layers:
        n += sum(x[0] * x[1] for x in s.mixer.tensor_shapes("", cfg.d_model).values() if len(x) == 2)
        m = s.mlp
        n += 0 if m is None else cfg.d_model * (3 * m.ff * m.top if hasattr(m, "top") else (3 if m.gated else 2) * m.ff)
    return n


def _vafodra(s) -> LayeredConfig:
    order = ORDER.replace("a", "p").replace("r", "d")
    left = dict(heads=s["H"], kv_heads=s["G"], dim=s["dk"], vdim=s["dk"], scale=s["dk"] ** -0.5)
    right = dict(heads=s["right"]["inner"] // 64, vdim=64, state=128, groups=8, norm_groups=8, conv=4)
    delta = dict(heads=s["H"], kv_heads=s["H"], dim=s["dk"], vdim=s["dk"], conv=4)

    def build(ff):
        return LayeredConfig(vocab_size=s["vocab"], d_model=s["d"], arch="Vafodra", seq_len=16384,
                             layers=hybrid_layers(order, left, right, delta, dict(p=ff, d=ff)))
    rest = _passed(_seredra(s)) - _passed(build(64))
    return build(max(64, 64 + rest // (3 * s["d"] * len(order)) // 64 * 64))


def kernels(s, T: int = 8192, L: int = 4096, B: int = 64, ctx: int = 4000, iters: int = 10) -> dict:
    """Kernel -> {ms, fraction of the roofline, the like kernel and its fraction}."""
    hbm, flops = _peaks()
    bf, f32 = torch.bfloat16, torch.float32
    d, H, G, dk, E, k, ff, F = (s[x] for x in ("d", "H", "G", "dk", "E", "top", "ffe", "ff"))
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    rnd = lambda *sh, dtype=bf: torch.randn(*sh, device="cuda", dtype=f32).mul_(0.5).to(dtype)
    one = lambda *sh: torch.ones(*sh, device="cuda")
    scale = dk ** -0.5
    out = {}

    def row(name, fn, roof_s, like=None):
        ms = _time(fn, iters, flush=flush)
        e = {"ms": round(ms, 4), "of_roofline": round(roof_s * 1e3 / ms, 3)}
        if like is not None:
            lname, lfn, lroof = like
            lms = _time(lfn, iters, flush=flush)
            e["like"] = {"kernel": lname, "ms": round(lms, 4), "of_roofline": round(lroof * 1e3 / lms, 3)}
            e["times_further"] = round((lroof / lms) / (roof_s / ms), 2)
        out[name] = e

    # ---- attention
    q, kk, vv, gate = rnd(1, L, H, dk), rnd(1, L, G, dk), rnd(1, L, G, dk), rnd(L, H * dk)
    o = torch.empty_like(q)
    linear, capped = ScoreRule(30.0, distance_slopes(H, "cuda")), ScoreRule(30.0)
    log = ScoreRule(log_amount=one(H), log_rate=one(H) * 0.3)
    roof = 2.0 * H * L * (L + 1) * dk / flops
    flash = ("capped, linear bias, gate", lambda: attn_ops.prompt_attention(q, kk, vv, scale, o, linear, gate), roof)
    row(f"prompt attention {L}, capped", lambda: attn_ops.prompt_attention(q, kk, vv, scale, o, capped), roof, flash)
    row(f"prompt attention {L}, logarithmic bias", lambda: attn_ops.prompt_attention(q, kk, vv, scale, o, log), roof, flash)
    nb = B * (ctx + 15) // 16 + B
    kc, vc = rnd(nb, 16, G, dk), rnd(nb, 16, G, dk)
    per = (ctx + 15) // 16
    bt = torch.randperm(nb, device="cuda")[:B * per].view(B, per).to(torch.int32)
    ctxs = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
    qd, od, gd = rnd(B, H * dk), torch.empty(B, H * dk, dtype=bf, device="cuda"), rnd(B, H * dk)
    roof = 4.0 * B * ctx * G * dk / hbm
    paged = ("capped, linear bias, gate", lambda: paged_ops.paged_attention_decode(qd, kc, vc, bt, ctxs, scale, od, linear, gd), roof)
    row(f"decode attention {B} at {ctx}, capped", lambda: paged_ops.paged_attention_decode(qd, kc, vc, bt, ctxs, scale, od, capped), roof, paged)
    row(f"decode attention {B} at {ctx}, logarithmic bias", lambda: paged_ops.paged_attention_decode(qd, kc, vc, bt, ctxs, scale, od, log), roof, paged)

    r, m = s["right"], s["ret"]
    inner, n, R = r["inner"], r["state"], r["dt_rank"]
    RH, rn, rv = m["heads"], m["dim"], m["vdim"]
    hs, ch = inner // 64, inner + 16 * 128
    for t, segs in ((T, [(i * (T // 4), T // 4, i, 0) for i in range(4)]), (T, [(0, T, 0, 0)]), (B, [(i, 1, i, 5) for i in range(B)])):
        tag = f"{t}" if len(segs) == t else f"{len(segs)} x {t // len(segs)}"
        seg = rc.Segments.of(segs, "cuda")
        # ---- recurrent mixers
        xbc, sdt, st = rnd(t, ch), rnd(t, hs, dtype=f32), torch.zeros(B, hs, 128, 64, device="cuda")
        states = 8.0 * len(segs) * hs * 128 * 64
        kw = dict(dt_bias=one(hs) * -3, a_log=one(hs), D=one(hs), state=st, heads=hs, groups=8, vdim=64, n=128, seg=seg)
        like = ("state space", lambda: rc.state_space(xbc, sdt, **kw), (2.0 * t * (ch + inner) + states + 4.0 * t * hs) / hbm)
        x, z, dt, low, y = rnd(t, inner), rnd(t, inner), rnd(t, inner, dtype=f32), rnd(t, R + 2 * n), torch.empty(t, inner, dtype=bf, device="cuda")
        A, D, db, ss = -one(inner, n), one(inner), one(inner) * -3, torch.zeros(B, inner, rc.up4(n), device="cuda")
        moved = t * inner * 10.0 + 4.0 * t * n + 8.0 * len(segs) * inner * n + 4.0 * inner * n
        row(f"selective scan {tag}", lambda: rc.selective_scan(x, dt, low[:, R:R + n], low[:, R + n:], z, A=A, D=D, dt_bias=db, state=ss, seg=seg, out=y),
            max(moved / hbm, t * inner * n / EXPONENTIALS), like)
        vkq, dec, rs = rnd(t, RH * (rv + 2 * rn)), torch.tensor(_decays(RH), device="cuda"), torch.zeros(B, RH, rn, rv, device="cuda")
        row(f"retention {tag}", lambda: rc.state_space(vkq, decay=dec, state=rs, heads=RH, groups=RH, vdim=rv, n=rn, seg=seg),
            (4.0 * t * RH * (rv + rn) + 8.0 * len(segs) * RH * rn * rv) / hbm, like)
        if len(segs) == 1:
            continue
        conv = lambda c, silu: (rnd(t, c), rnd(c, 4, dtype=f32), torch.zeros(B, 3, c, dtype=bf, device="cuda"), silu)
        cost = lambda c: (4.0 * t * c + 12.0 * len(segs) * c) / hbm
        cx = conv(ch, True)
        clike = ("short convolution (state space)", lambda: rc.short_conv(cx[0], cx[1], None, cx[2], seg), cost(ch))
        for name, c, silu in (("scan", inner, True), ("queries, keys, values", (H + 2 * G) * dk, False)):
            a = conv(c, silu)
            row(f"short convolution ({name}) {t}", lambda: rc.short_conv(a[0], a[1], None, a[2], seg, silu=silu), cost(c), clike)
        # ---- positions, norms of queries and keys
        qkv, g16, gq, gk = rnd(t, (H + 2 * G) * dk), rnd(dk), rnd(H * dk, dtype=f32), rnd(G * dk, dtype=f32)
        slots, pos = torch.randperm(nb * 16, device="cuda")[:t], torch.arange(t, device="cuda")
        hp = dict(eps=1e-5, k_cache=kc, v_cache=vc, slots=slots)
        # read and write queries and keys, read values, store both
        moved = 2.0 * t * dk * (2 * H + 2 * G + G + 2 * G)
        hlike = ("head norms + append", lambda: head_prep_(qkv, H, G, dk, dk, q_gamma=g16, k_gamma=g16, **hp), moved / hbm)
        row(f"row norms + temperature + append {t}", lambda: row_prep_(qkv, H, G, dk, dk, q_gamma=gq, k_gamma=gk, pos=pos, temp_coef=0.1, temp_every=4096, **hp),
            moved / hbm, hlike)
        table = rope_ops.rotary_table(pos, torch.tensor(RotarySpec(dk, 500000.0).frequencies(), dtype=torch.float64, device="cuda"))
        row(f"head norms + rotation + append, keys as values {t}", lambda: head_prep_(qkv, H, G, dk, dk, q_gamma=g16, k_gamma=g16, rot=table, half=True,
                                                                                     values_are_keys=True, **hp),
            (2.0 * t * dk * (2 * H + 2 * G + G + 2 * G) + 4.0 * t * dk) / hbm, hlike)
        rtable = rope_ops.rotary_table(pos, torch.tensor(RotarySpec(rn, 10000.0).frequencies(), dtype=torch.float64, device="cuda"))
        row(f"rotation (retention) {t}", lambda: head_prep_(vkq, RH, RH, rn, rn, rot=rtable, half=True, k_scale=0.1, q_col=RH * (rv + rn), k_col=RH * rv),
            (8.0 * t * RH * rn + 4.0 * t * rn) / hbm, ("rope", lambda: rope_ops.rope_(qkv, H + G, dk, positions=pos), 4.0 * t * dk * (H + G) / hbm))
        # ---- norms
        ry, rz, w = rnd(t, RH * rv), rnd(t, RH * rv), one(dk)
        dy, dz = rnd(t, H * dk), rnd(t, H * dk)
        row(f"norm per head + gate {t}", lambda: rc.gated_norm(ry, rz, None, RH, 1e-5, False, out=ry), 6.0 * t * RH * rv / hbm,
            ("gated norm per head (delta rule)", lambda: rc.gated_norm(dy, dz, w, H, 1e-5, False, out=dy), 6.0 * t * H * dk / hbm))
        yf, xs, h, wd = rnd(t, d, dtype=f32), rnd(t, d, dtype=f32), rnd(t, d), rnd(d, dtype=f32)
        row(f"residual + norm {t}", lambda: norm_ops.residual_norm(yf, None, None, 1e-5, True, x=xs, h=h, next_gamma=wd), 14.0 * t * d / hbm,
            ("norm + residual + norm", lambda: norm_ops.residual_norm(yf, wd, None, 1e-5, True, x=xs, h=h, next_gamma=wd), 14.0 * t * d / hbm))
        # ---- routed feed-forward
        logits = rnd(t, E, dtype=f32)
        row(f"router choice {t}", lambda: moe_ops.route_sigmoid(logits, k), 4.0 * t * (E + 2 * k) / hbm,
            ("group-limited sigmoid choice", lambda: moe_ops.route_sigmoid(logits, k, 4, 2, None, 2), 4.0 * t * (E + 2 * k) / hbm))
        idx, rw = moe_ops.route_sigmoid(logits, k)
        pl = moe_ops.plan(idx, E)
        gu = rnd(pl.max_rows, 2 * ff)
        row(f"weighted swiglu {t}", lambda: moe_ops.swiglu_rows(gu, pl, weights=rw), 6.0 * t * k * ff / hbm,
            ("expert swiglu", lambda: moe_ops.swiglu_rows(gu, pl), 6.0 * t * k * ff / hbm))
        yp = rnd(pl.max_rows, d)
        row(f"experts' sum + residual + norm {t}", lambda: norm_ops.residual_norm(yp, None, None, 1e-5, True, x=xs, h=h, next_gamma=wd, routed=(pl.slot_pos, None)),
            t * d * (2.0 * k + 10) / hbm, ("combine + norm + residual + norm", lambda: norm_ops.residual_norm(
                yp, wd, None, 1e-5, True, x=xs, h=h, next_gamma=wd, routed=(pl.slot_pos, rw)), t * d * (2.0 * k + 10) / hbm))
        del gu, yp, xbc, x, z, dt, y, vkq, ry, rz

        # ---- products, beside one of Vafodra's of about the shape
        def product(name, n_, k_, ln, lk, **kw):
            a, b = rnd(t, k_), rnd(n_, k_)
            la, lb = rnd(t, lk), rnd(ln, lk)
            ob = 4 if kw.get("out_dtype") is f32 else 2
            time = lambda n_, k_, o_: max(2.0 * t * n_ * k_ / flops, (2.0 * (n_ * k_ + t * k_) + o_ * t * n_) / hbm)
            row(f"{name} {t}", lambda: gemm(a, b, **kw), time(n_, k_, ob), (f"product {lk} -> {ln}", lambda: gemm(la, lb), time(ln, lk, 2)))
        product("packed projection with bias", (H + 2 * G) * dk, d, (H + 2 * G) * dk, d, bias=rnd((H + 2 * G) * dk))
        product("packed projection (parallel)", (H + G) * dk + 2 * inner, d, (H + 2 * G) * dk + inner + ch, d)
        product("packed projection (retention)", 2 * RH * (rn + rv), d, (H + 2 * G) * dk + inner + ch, d)
        product("step sizes, B and C", R + 2 * n, inner, hs, d)
        product("step sizes", inner, R, hs, d, out_dtype=f32)
        product("joined output", d, H * dk + inner, d, inner, out_dtype=f32)
        product("output with bias", d, H * dk, d, H * dk, bias=rnd(d), out_dtype=f32)
        product("up + squared relu", F, d, 2 * F, d, act="relu2")
    return out


def run(sizes=None, with_kernels: bool = True) -> dict:
    out = {"metric": "decoder_serving", "dtype": "bf16", "data": "synthetic: random weights and token ids",
           "l2": "kernels: flushed before every launch (256 MiB write); model steps: weights and cache exceed L2", "sizes": {}}
    for name in sizes or SIZES:
        s = SIZES[name]
        both = {"seredra": _seredra(s), "vafodra": _vafodra(s)}
        e = {"config": {**s, "order": ORDER, "kv_from": KV_FROM, "dense": DENSE}, "weights_passed": {m: _passed(c) for m, c in both.items()}}
        for model, c in both.items():
            e[model] = throughput(c)
            torch.cuda.empty_cache()
        if with_kernels:
            e["kernels"] = kernels(s)
            torch.cuda.empty_cache()
        out["sizes"][name] = e
    return out
