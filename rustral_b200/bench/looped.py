"""Serving throughput of the looped decoder (Bikilix) beside the layered one with routed experts (Dolurax) at equal size, and its
kernels beside the like kernels of the other models against the measured roofline.

    python bench.py --decoders bikilix                 # all sizes, JSON line
    python bench.py --decoders bikilix --decoder-size medium

Both models have random weights, the same width, attention heads, head size and vocabulary, as many layers that run (a layer in the
loop counts once per pass) and the same feed-forward work per token (Dolurax: `top` experts and a shared one; Bikilix: one expert more).
Timing as in bench.decoders.  The like kernel is Dolurax's for the routed feed-forward and the plain one of the Llama-style model
(no cap, no bias, no gate) for attention, positions, norms and products.
"""
from __future__ import annotations

import torch

from ..models.layered import LayeredConfig, LoopSpec, RotarySpec, sandwich_layers
from ..ops import attention as attn_ops
from ..ops import latent as latent_ops
from ..ops import moe as moe_ops
from ..ops import norm as norm_ops
from ..ops import paged as paged_ops
from ..ops import rotary as rope_ops
from ..ops.attention import ScoreRule
from ..ops.heads import head_prep_
from ..ops.matmul import gemm
from .decoders import SIZES as DOLURAX_SIZES
from .decoders import _layered as _dolurax
from .decoders import _peaks, _time, throughput

ORDER, DENSE = "wwlwlw", (0,)
SIZES = {
    "small": dict(window=1024, rot=64, loop=(2, 4, 2), latent=dict(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=768)),
    "medium": dict(window=2048, rot=64, loop=None, latent=dict(heads=32, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=1536)),
    "head64": dict(window=512, rot=32, loop=(2, 4, 2), latent=dict(heads=32, dim=64, rot_dim=32, vdim=64, kv_rank=256, q_rank=768)),
}
SIZES = {name: {**DOLURAX_SIZES[name], **s} for name, s in SIZES.items()}
YARN = dict(base=500000.0, factor=8.0, original=4096, fast=32.0, slow=1.0, scaled=True)


def _bikilix(s) -> LayeredConfig:
    order = ORDER[:s["layers"]]
    att = dict(heads=s["H"], kv_heads=s["G"], dim=s["dk"], vdim=s["dk"], scale=s["dk"] ** -0.5, window=s["window"], rot=dict(dims=s["rot"], base=500000.0))
    m = s["latent"]
    lat = dict(m, scale=(m["dim"] + m["rot_dim"]) ** -0.5, rot=dict(dims=m["rot_dim"], **YARN))
    return LayeredConfig(vocab_size=s["vocab"], d_model=s["d"], arch="Bikilix", seq_len=16384, loop=LoopSpec(*s["loop"]) if s["loop"] else None,
                         layers=sandwich_layers(order, att, lat, (s["top"] + 1) * s["ff"],
                                                dict(ff=s["ff"], experts=s["E"], top=s["top"] + 1, groups=4, keep=2, limit=7.0), DENSE))


def kernels(s, T: int = 8192, L: int = 4096, B: int = 64, ctx: int = 4000, iters: int = 10) -> dict:
    """Kernel -> {ms, fraction of the roofline, the like kernel and its fraction}."""
    hbm, flops = _peaks()
    bf, f32 = torch.bfloat16, torch.float32
    d, H, G, dk, E, k, ff = (s[x] for x in ("d", "H", "G", "dk", "E", "top", "ff"))
    F, k1 = (k + 1) * ff, k + 1
    m = s["latent"]
    HL, dn, dr, dv, R, Q = (m[x] for x in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
    W = R + dr
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    rnd = lambda *sh, dtype=bf: torch.randn(*sh, device="cuda", dtype=f32).mul_(0.5).to(dtype)
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
    q, kk, vv = rnd(1, L, H, dk), rnd(1, L, G, dk), rnd(1, L, G, dk)
    o = torch.empty_like(q)
    flash = ("flash forward", lambda: attn_ops.attention_forward(q, kk, vv, True, scale, out=o, want_lse=False), 2.0 * H * L * (L + 1) * dk / flops)
    for window in (s["window"], 0):
        seen = sum(min(i + 1, window or L) for i in range(L))
        rule = ScoreRule(window=window) if window else None
        row(f"prompt attention {L}" + (f", window {window}" if window else ", no window"), lambda: attn_ops.prompt_attention(q, kk, vv, scale, o, rule),
            4.0 * H * seen * dk / flops, flash)
    ql, kv, kr, gl = rnd(1, L, HL, dn + dr), rnd(L, HL * (dn + dv)), rnd(L, W), rnd(L, HL * dv)
    ol = torch.empty(1, L, HL, dv, dtype=bf, device="cuda")
    row(f"latent prompt attention {L}", lambda: attn_ops.prompt_attention_split(ql, kv[:, :HL * dn].view(1, L, HL, dn), kv[:, HL * dn:].view(1, L, HL, dv), kr[:, R:],
                                                                                0.1, ol, gate=gl), 1.0 * HL * L * (L + 1) * (dn + dr + dv) / flops, flash)
    nb = B * (ctx + 15) // 16 + B
    kc, vc = rnd(nb, 16, G, dk), rnd(nb, 16, G, dk)
    per = (ctx + 15) // 16
    bt = torch.randperm(nb, device="cuda")[:B * per].view(B, per).to(torch.int32)
    ctxs = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
    short = torch.full((B,), s["window"], dtype=torch.int32, device="cuda")
    qd, od = rnd(B, H * dk), torch.empty(B, H * dk, dtype=bf, device="cuda")
    roof = 4.0 * B * s["window"] * G * dk / hbm
    win = ScoreRule(window=s["window"])
    row(f"decode attention {B} at {ctx}, window {s['window']}", lambda: paged_ops.paged_attention_decode(qd, kc, vc, bt, ctxs, scale, od, win), roof,
        ("paged decode of as many keys", lambda: paged_ops.paged_attention_decode(qd, kc, vc, bt, short, scale, od), roof))
    paged = ("paged decode", lambda: paged_ops.paged_attention_decode(qd, kc, vc, bt, ctxs, scale, od), 4.0 * B * ctx * G * dk / hbm)
    cache, qa = rnd(nb, 16, 1, W), rnd(B, HL * W)
    row(f"latent decode attention {B} at {ctx}", lambda: latent_ops.latent_decode(qa, cache, R, bt, ctxs, 0.05),
        max(2.0 * B * ctx * W / hbm, 2.0 * B * HL * ctx * (W + R) / flops), paged)

    pos_f = torch.tensor(RotarySpec(dr, **YARN).frequencies(), dtype=torch.float64, device="cuda")
    att_f = torch.tensor(RotarySpec(s["rot"], 500000.0).frequencies(), dtype=torch.float64, device="cuda")
    for t in (T, B):
        qkv = rnd(t, (H + 2 * G) * dk)
        slots, pos = torch.randperm(nb * 16, device="cuda")[:t], torch.arange(t, device="cuda")

        def rope():
            rope_ops.rope_(qkv, H + G, dk, positions=pos)
            paged_ops.kv_append(qkv[:, H * dk:(H + G) * dk], qkv[:, (H + G) * dk:], kc, vc, slots)
        ropes = ("rope + append", rope, 2.0 * t * dk * (2 * H + 2 * G + 4 * G) / hbm)
        table, ltable = rope_ops.rotary_table(pos, att_f), rope_ops.rotary_table(pos, pos_f)
        # ---- positions, latents
        row(f"rotation + append {t}", lambda: head_prep_(qkv, H, G, dk, dk, k_cache=kc, v_cache=vc, slots=slots, rot=table),
            (4.0 * t * s["rot"] * H + 2.0 * t * G * (dk + s["rot"]) + 2.0 * t * G * (dk + 2 * dk) + 4.0 * t * s["rot"]) / hbm, ropes)
        z, gq, gk = rnd(t, Q + W + HL * dv), rnd(Q, dtype=f32), rnd(R, dtype=f32)
        row(f"latent norms + rotation + append {t}", lambda: latent_ops.latent_prep_(z, 0, Q, Q, R, dr, q_gamma=gq, kv_gamma=gk, eps=1e-5, table=ltable, cache=cache,
                                                                                     slots=slots), (4.0 * t * (Q + W) + 2.0 * t * W + 4.0 * t * dr) / hbm, ropes)
        ql = rnd(t, HL * (dn + dr))
        wkv = rnd(HL * (dn + dv), R)
        like = None
        if t == T:
            row(f"query rotation {t}", lambda: rope_ops.rotate_pairs_(ql, HL, dn + dr, dn, ltable), (4.0 * t * HL * dr + 4.0 * t * dr) / hbm,
                ("rope", lambda: rope_ops.rope_(qkv, H + G, dk, positions=pos), 4.0 * t * dk * (H + G) / hbm))
        else:
            ow = rnd(H * dk, d)
            like = ("output projection of one token each", lambda: gemm(od, ow, b_mn=True), 2.0 * (H * dk * d + t * (d + H * dk)) / hbm)
            row(f"query x key product + rotation {t}", lambda: latent_ops.head_product(ql, dn + dr, wkv[:HL * dn], HL, R, dn, transposed=True, tail=dr, table=ltable),
                2.0 * (HL * dn * R + t * HL * (dn + dr + W)) / hbm, like)
            c, gate = rnd(t, HL * R), rnd(t, HL * dv)
            row(f"value product + gate {t}", lambda: latent_ops.head_product(c, R, wkv[HL * dn:], HL, dv, R, transposed=False, gate=gate),
                2.0 * (HL * dv * R + t * HL * (R + 2 * dv)) / hbm, like)
        # ---- norms
        y, x, h, w, g16 = rnd(t, d, dtype=f32), rnd(t, d, dtype=f32), rnd(t, d), rnd(d, dtype=f32), rnd(d)
        nl = ("rms norm", lambda: norm_ops.norm_forward(h, g16, None, 1e-5, True, want_stats=False), 4.0 * t * d / hbm)
        row(f"norm + residual + norm {t}", lambda: norm_ops.residual_norm(y, w, None, 1e-5, True, x=x, h=h, next_gamma=w), 14.0 * t * d / hbm, nl)
        # ---- routed feed-forward
        logits, corr = rnd(t, E, dtype=f32), rnd(E, dtype=f32)
        row(f"router choice {t}", lambda: moe_ops.route_sigmoid(logits, k1, 4, 2, corr, 2), 4.0 * t * (E + 2 * k1) / hbm,
            ("group-limited softmax choice", lambda: moe_ops.route_groups(logits, k, 4, 2), 4.0 * t * (E + 2 * k) / hbm))
        idx, rw = moe_ops.route_sigmoid(logits, k1, 4, 2, None, 2)
        pl = moe_ops.plan(idx, E)
        gu = rnd(pl.max_rows, 2 * ff)
        row(f"clamped gate {t}", lambda: moe_ops.swiglu_rows(gu, pl, "clamped", limit=7.0), 6.0 * t * k1 * ff / hbm,
            ("expert swiglu", lambda: moe_ops.swiglu_rows(gu, pl), 6.0 * t * k1 * ff / hbm))
        yp = rnd(pl.max_rows, d)
        row(f"combine + norm + residual + norm {t}", lambda: norm_ops.residual_norm(yp, w, None, 1e-5, True, x=x, h=h, next_gamma=w, routed=(pl.slot_pos, rw)),
            t * d * (2.0 * k1 + 10) / hbm, ("combine + norm + residual", lambda: norm_ops.residual_norm(yp, g16, g16, 1e-5, x=x, h=h, routed=(pl.slot_pos, rw), add=h),
                                            t * d * (2.0 * k1 + 12) / hbm))
        del gu, yp
        # ---- products

        def product(name, n, kk_, ln, lk, **kw):
            a, b = rnd(t, kk_), rnd(n, kk_)
            la, lb = rnd(t, lk), rnd(ln, lk)
            ob = 4 if kw.get("out_dtype") is f32 else 2
            time = lambda n_, k_, o_: max(2.0 * t * n_ * k_ / flops, (2.0 * (n_ * k_ + t * k_) + o_ * t * n_) / hbm)
            row(f"{name} {t}", lambda: gemm(a, b, **kw), time(n, kk_, ob), (f"product {lk} -> {ln}", lambda: gemm(la, lb), time(ln, lk, 2)))
        bias = rnd((H + 2 * G) * dk)
        product("packed projection with bias", (H + 2 * G) * dk, d, (H + 2 * G) * dk, d, bias=bias)
        product("packed projection (latent)", Q + W + HL * dv, d, (H + 2 * G) * dk, d)
        product("query product", HL * (dn + dr), Q, (H + 2 * G) * dk, d)
        if t == T:
            product("keys and values of all heads", HL * (dn + dv), R, (H + 2 * G) * dk, d)
        product("up + squared relu", F, d, 2 * F, d, act="relu2")
        product("loop input", d, 2 * d, d, H * dk, bias=rnd(d), out_dtype=f32)
    return out


def run(sizes=None, with_kernels: bool = True) -> dict:
    out = {"metric": "decoder_serving", "dtype": "bf16", "data": "synthetic: random weights and token ids",
           "l2": "kernels: flushed before every launch (256 MiB write); model steps: weights and cache exceed L2", "sizes": {}}
    for name in sizes or SIZES:
        s = SIZES[name]
        cfg = _bikilix(s)
        e = {"config": {**s, "order": ORDER[:s["layers"]], "runs": len(cfg.runs)}}
        for model, c in (("bikilix", cfg), ("dolurax", _dolurax({**s, "layers": len(cfg.runs)}))):
            e[model] = throughput(c)
            torch.cuda.empty_cache()
        if with_kernels:
            e["kernels"] = kernels(s)
            torch.cuda.empty_cache()
        out["sizes"][name] = e
    return out
