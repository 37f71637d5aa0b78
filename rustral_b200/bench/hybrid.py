"""Serving throughput of the hybrid decoder (Vafodra) beside the Llama-style decoder at equal size, and its kernels beside the
like kernels of that model against the measured roofline.

    python bench.py --decoders vafodra                 # all sizes, JSON line
    python bench.py --decoders vafodra --decoder-size medium

Both models have random weights, the same width, attention heads, head size and vocabulary, and the same number of parameters per
layer (the hybrid's feed-forward is narrower by what its other mixers take).  Timing as in bench.decoders.  The recurrent mixers
have no like kernel; they are set beside the attention kernels that do the same job, mixing over the sequence.
"""
from __future__ import annotations

import torch

from ..models.config import GPTConfig
from ..models.layered import LayeredConfig, hybrid_layers
from ..ops import attention as attn_ops
from ..ops import moe as moe_ops
from ..ops import norm as norm_ops
from ..ops import paged as paged_ops
from ..ops import recurrent as rc
from ..ops import rotary as rope_ops
from ..ops.attention import ScoreRule
from ..ops.heads import head_prep_
from ..ops.matmul import gemm
from .decoders import _peaks, _time, throughput

ORDER = "ppdpppdp"
SIZES = {
    "small": dict(d=2048, vocab=32768, layers=8, dense_ff=8192, window=1024, left=dict(heads=16, kv_heads=4, dim=128, vdim=128),
                  right=dict(heads=64, vdim=64, state=128, groups=8, norm_groups=8, conv=4),
                  delta=dict(heads=16, kv_heads=16, dim=128, vdim=128, conv=4), ff=dict(p=3328, d=6400)),
    "medium": dict(d=4096, vocab=65536, layers=4, dense_ff=14336, window=2048, left=dict(heads=32, kv_heads=8, dim=128, vdim=128),
                   right=dict(heads=128, vdim=64, state=128, groups=8, norm_groups=8, conv=4),
                   delta=dict(heads=32, kv_heads=16, dim=128, vdim=128, conv=4), ff=dict(p=5376, d=12288)),
    "head64": dict(d=2048, vocab=32768, layers=8, dense_ff=8192, window=512, left=dict(heads=32, kv_heads=8, dim=64, vdim=64),
                   right=dict(heads=32, vdim=128, state=64, groups=4, norm_groups=1, conv=4),
                   delta=dict(heads=32, kv_heads=32, dim=64, vdim=64, conv=4), ff=dict(p=3584, d=6400)),
}
KEEP = 4


def _hybrid(s) -> LayeredConfig:
    left = dict(s["left"], scale=s["left"]["dim"] ** -0.5, window=s["window"], keep_first=KEEP)
    return LayeredConfig(vocab_size=s["vocab"], d_model=s["d"], arch="Vafodra", embed_scale=1.0, residual_mult=0.5, seq_len=16384,
                         layers=hybrid_layers(ORDER[:s["layers"]], left, s["right"], s["delta"], s["ff"]))


def _llama(s) -> GPTConfig:
    return GPTConfig(vocab_size=s["vocab"], seq_len=16384, n_layer=s["layers"], n_head=s["left"]["heads"],
                     n_kv_head=s["left"]["kv_heads"], d_model=s["d"], ffn_dim=s["dense_ff"], arch="llama")


def kernels(s, T: int = 8192, L: int = 4096, B: int = 64, ctx: int = 4000, iters: int = 10) -> dict:
    """Kernel -> {ms, fraction of the roofline, the like kernel of the Llama-style model and its fraction}."""
    hbm, flops = _peaks()
    bf, f32 = torch.bfloat16, torch.float32
    d, F = s["d"], s["dense_ff"]
    H, G, dk = s["left"]["heads"], s["left"]["kv_heads"], s["left"]["dim"]
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    rnd = lambda *sh, dtype=bf: torch.randn(*sh, device="cuda", dtype=f32).mul_(0.5).to(dtype)
    rule = ScoreRule(window=s["window"], keep_first=KEEP, sink=True)
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
    q, kk, vv, hg = rnd(1, L, H, dk), rnd(1, L, G, dk), rnd(1, L, G, dk), rnd(L, H, dtype=f32)
    o = torch.empty_like(q)
    seen = sum(min(i + 1, s["window"] + KEEP) for i in range(L))
    flash = ("flash forward", lambda: attn_ops.attention_forward(q, kk, vv, True, scale, out=o, want_lse=False), 2.0 * H * L * (L + 1) * dk / flops)
    row(f"prompt attention {L}", lambda: attn_ops.prompt_attention(q, kk, vv, scale, o, rule, head_gate=hg), 4.0 * H * seen * dk / flops, flash)
    nb = B * (ctx + 15) // 16 + B
    kc, vc = rnd(nb, 16, G, dk), rnd(nb, 16, G, dk)
    per = (ctx + 15) // 16
    bt = torch.randperm(nb, device="cuda")[:B * per].view(B, per).to(torch.int32)
    ctxs = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
    short = torch.full((B,), s["window"] + KEEP, dtype=torch.int32, device="cuda")
    qd, hd, od = rnd(B, H * dk), rnd(B, H, dtype=f32), torch.empty(B, H * dk, dtype=bf, device="cuda")
    roof = 4.0 * B * (s["window"] + KEEP) * G * dk / hbm
    paged = ("paged decode of as many keys", lambda: paged_ops.paged_attention_decode(qd, kc, vc, bt, short, scale, od), roof)
    row(f"decode attention {B} at {ctx}", lambda: paged_ops.paged_attention_decode(qd, kc, vc, bt, ctxs, scale, od, rule, head_gate=hd), roof, paged)

    r, m = s["right"], s["delta"]
    inner, ch = r["heads"] * r["vdim"], r["heads"] * r["vdim"] + 2 * r["groups"] * r["state"]
    dch, dvn = 2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"], m["heads"] * m["vdim"]
    one = lambda *sh: torch.ones(*sh, device="cuda")
    for t, segs in ((T, [(i * (T // 4), T // 4, i, 0) for i in range(4)]), (T, [(0, T, 0, 0)]), (B, [(i, 1, i, 5) for i in range(B)])):
        tag = f"{t}" if len(segs) == t else f"{len(segs)} x {t // len(segs)}"
        seg = rc.Segments.of(segs, "cuda")
        decode = t == B
        like = ("paged decode", lambda: paged_ops.paged_attention_decode(qd, kc, vc, bt, ctxs, scale, od), 4.0 * B * ctx * G * dk / hbm) if decode else flash
        qkv = rnd(t, (H + 2 * G) * dk)
        slots, pos = torch.randperm(nb * 16, device="cuda")[:t], torch.arange(t, device="cuda")

        def rope():
            rope_ops.rope_(qkv, H + G, dk, positions=pos)
            paged_ops.kv_append(qkv[:, H * dk:(H + G) * dk], qkv[:, (H + G) * dk:], kc, vc, slots)
        ropes = ("rope + append", rope, 2.0 * t * dk * (2 * H + 2 * G + 4 * G) / hbm)
        # ---- recurrent mixers
        xbc, dt, st = rnd(t, ch), rnd(t, r["heads"], dtype=f32), torch.zeros(B, r["heads"], r["state"], r["vdim"], device="cuda")
        states = 8.0 * len(segs) * r["heads"] * r["state"] * r["vdim"]
        kw = dict(dt_bias=one(r["heads"]) * -3, a_log=one(r["heads"]), D=one(r["heads"]), state=st, heads=r["heads"], groups=r["groups"],
                  vdim=r["vdim"], n=r["state"], seg=seg)
        row(f"state space {tag}", lambda: rc.state_space(xbc, dt, **kw), (2.0 * t * (ch + inner) + states + 4.0 * t * r["heads"]) / hbm, like)
        dq, ab, ds = rnd(t, dch), rnd(t, 2 * m["heads"], dtype=f32), torch.zeros(B, m["heads"], m["dim"], m["vdim"], device="cuda")
        states = 8.0 * len(segs) * m["heads"] * m["dim"] * m["vdim"]
        dw = dict(dt_bias=one(m["heads"]) * -3, a_log=one(m["heads"]), state=ds, heads=m["heads"], kv_heads=m["kv_heads"], dk=m["dim"],
                  dv=m["vdim"], seg=seg)
        row(f"delta rule {tag}", lambda: rc.delta_rule(dq, ab[:, :m["heads"]], ab[:, m["heads"]:], **dw),
            (2.0 * t * (dch + dvn) + states + 8.0 * t * m["heads"]) / hbm, like)
        if len(segs) == 1:
            continue
        cw, cb, cs = rnd(ch, 4, dtype=f32), rnd(ch, dtype=f32), torch.zeros(B, 3, ch, dtype=bf, device="cuda")
        row(f"short convolution {t}", lambda: rc.short_conv(xbc, cw, cb, cs, seg), (4.0 * t * ch + 12.0 * len(segs) * ch) / hbm, ropes)
        y, z, w = rnd(t, inner), rnd(t, inner), one(inner)
        h, g = rnd(t, d), rnd(d)
        nl = ("rms norm", lambda: norm_ops.norm_forward(h, g, None, 1e-5, True, want_stats=False), 4.0 * t * d / hbm)
        row(f"gated norm, {r['norm_groups']} parts {t}", lambda: rc.gated_norm(y, z, w, r["norm_groups"], 1e-5, True, out=y), 6.0 * t * inner / hbm, nl)
        dy, dz, dwt = rnd(t, dvn), rnd(t, dvn), one(m["vdim"])
        row(f"gated norm per head {t}", lambda: rc.gated_norm(dy, dz, dwt, m["heads"], 1e-5, False, out=dy), 6.0 * t * dvn / hbm, nl)
        row(f"append {t}", lambda: head_prep_(qkv, H, G, dk, dk, k_cache=kc, v_cache=vc, slots=slots), 2.0 * t * dk * 4 * G / hbm, ropes)
        # ---- norms, feed-forward, products
        x, wd, dyt = rnd(t, d, dtype=f32), one(d), (one(d), one(d), one(1))
        ys = [rnd(t, d) for _ in range(3)]
        row(f"norms + residual + dynamic tanh {t}", lambda: norm_ops.stream_update(x, a=ys[0], wa=wd, b=ys[1], wb=wd, c=ys[2], normed=0.5, mult=0.5, dyt=dyt, h=h),
            16.0 * t * d / hbm, nl)
        row(f"residual + dynamic tanh {t}", lambda: norm_ops.stream_update(x, c=ys[0], mult=0.5, dyt=dyt, h=h), 12.0 * t * d / hbm, nl)
        ff = s["ff"]["p"]
        gu, gl = rnd(t, 2 * ff), rnd(t, 2 * F)
        row(f"relu(gate) * up {t}", lambda: moe_ops.swiglu_rows(gu, act="relu"), 6.0 * t * ff / hbm,
            ("swiglu", lambda: rope_ops.swiglu_forward(gl), 6.0 * t * F / hbm))
        del gu, gl, x, ys, y, z

        def product(name, n, k, ln, lk):
            a, b = rnd(t, k), rnd(n, k)
            la, lb = rnd(t, lk), rnd(ln, lk)
            time = lambda n_, k_: max(2.0 * t * n_ * k_ / flops, 2.0 * (n_ * k_ + t * (n_ + k_)) / hbm)
            row(f"{name} {t}", lambda: gemm(a, b), time(n, k), ("dense gate + up" if ln != d else "dense down", lambda: gemm(la, lb), time(ln, lk)))
        product("packed projection (parallel)", (H + 2 * G) * dk + inner + ch + 2 * ff, d, 2 * F, d)
        product("packed projection (delta)", dch + dvn + 2 * s["ff"]["d"], d, 2 * F, d)
        product("state-space output", d, inner, d, F)
        product("delta + feed-forward output", d, dvn + s["ff"]["d"], d, F)
        del xbc, dq
    return out


def run(sizes=None, with_kernels: bool = True) -> dict:
    out = {"metric": "decoder_serving", "dtype": "bf16", "data": "synthetic: random weights and token ids",
           "l2": "kernels: flushed before every launch (256 MiB write); model steps: weights and cache exceed L2", "sizes": {}}
    for name in sizes or SIZES:
        s = SIZES[name]
        e = {"config": {**s, "order": ORDER[:s["layers"]], "keep_first": KEEP}}
        for model, cfg in (("vafodra", _hybrid(s)), ("llama", _llama(s))):
            e[model] = throughput(cfg)
            torch.cuda.empty_cache()
        e["parameters"] = {"vafodra": _hybrid(s).num_parameters(), "llama": _llama(s).num_parameters()}
        if with_kernels:
            e["kernels"] = kernels(s)
            torch.cuda.empty_cache()
        out["sizes"][name] = e
    return out
