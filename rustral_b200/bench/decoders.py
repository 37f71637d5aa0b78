"""Serving throughput of the layered decoder (Dolurax) beside the Llama-style decoder at equal size, and the same comparison
kernel by kernel against the measured roofline.

    python bench.py --decoders                 # all sizes, JSON line
    python bench.py --decoders --decoder-size medium

Both models have random weights, the same width, heads, head size and vocabulary, and the same feed-forward work per token
(chosen experts + shared expert = the dense hidden size).  Prefill: prompts in one step of the runner; decode: the runner's
graphed step at a given context.  Device time by CUDA events; kernels are timed one by one with the L2 cache flushed before
every launch.
"""
from __future__ import annotations

import json
import os
import statistics

import torch

from .. import ops
from ..models.config import GPTConfig
from ..models.layered import LayeredConfig, uniform_layers
from ..ops import attention as attn_ops
from ..ops import moe as moe_ops
from ..ops import norm as norm_ops
from ..ops import paged as paged_ops
from ..ops import rotary as rope_ops
from ..ops.attention import ScoreRule, distance_slopes
from ..ops.heads import head_prep_
from ..ops.matmul import gemm
from ..serve.model_runner import ModelRunner
from ..models.registry import build_weights

# width, heads, kv heads, head size, experts, chosen, hidden size of an expert (chosen + 1 shared = the dense one), layers
SIZES = {
    "small": dict(d=2048, H=16, G=4, dk=128, E=32, top=3, ff=2048, layers=8, vocab=32768),
    "medium": dict(d=4096, H=32, G=8, dk=128, E=32, top=7, ff=1792, layers=4, vocab=65536),
    "head64": dict(d=2048, H=32, G=8, dk=64, E=64, top=7, ff=1024, layers=8, vocab=32768),
}
CHUNK = 4096


def _peaks() -> tuple:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            p = json.load(f)
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12
    except OSError:
        return 6.65e12, 1.59e15


def _layered(s) -> LayeredConfig:
    return LayeredConfig(vocab_size=s["vocab"], d_model=s["d"], logit_softcap=30.0, seq_len=16384, layers=uniform_layers(
        s["layers"], dict(heads=s["H"], kv_heads=s["G"], dim=s["dk"], vdim=s["dk"], scale=s["dk"] ** -0.5, softcap=30.0, chunk=CHUNK,
                          v_mix=True),
        dict(ff=s["ff"], experts=s["E"], top=s["top"], groups=4, keep=2, shared_ff=s["ff"])))


def _llama(s) -> GPTConfig:
    return GPTConfig(vocab_size=s["vocab"], seq_len=16384, n_layer=s["layers"], n_head=s["H"], n_kv_head=s["G"], d_model=s["d"],
                     ffn_dim=(s["top"] + 1) * s["ff"], arch="llama")


def _time(fn, iters: int, warmup: int = 3, flush=None) -> float:
    """Median milliseconds of one call."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    ev = []
    for _ in range(iters):
        if flush is not None:
            flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        ev.append((a, b))
    torch.cuda.synchronize()
    return statistics.median(a.elapsed_time(b) for a, b in ev)


def throughput(cfg, prompts=((4, 2048), (1, 8192)), decodes=((1, 2048), (32, 2048), (64, 4000)), iters: int = 8) -> dict:
    runner = ModelRunner(cfg, params=build_weights(cfg, "cuda"), device="cuda", num_blocks=64 * 4096 // 16 + 64, block_size=16,
                         num_slots=max(B for B, _ in decodes))
    g = torch.Generator().manual_seed(0)
    out = {}
    for n, L in prompts:
        toks = [torch.randint(0, cfg.vocab_size, (L,), generator=g).tolist() for _ in range(n)]
        for i in range(n):
            assert runner.cache.allocate(i, L)
        ms = _time(lambda: runner.step_mixed([(i, toks[i], 0, True) for i in range(n)], [], [], []), iters)
        out[f"prefill {n} x {L}"] = {"ms": round(ms, 3), "tokens_per_s": round(n * L / ms * 1e3)}
        for i in range(n):
            runner.cache.free(i)
    for B, ctx in decodes:
        for i in range(B):
            assert runner.cache.allocate(i, ctx)
        ids, lens = list(range(B)), [ctx] * B
        tok = torch.randint(0, cfg.vocab_size, (B,), generator=g).tolist()
        runner.decode(ids, tok, lens)                                   # captures the graph
        (gr,) = [v for k, v in runner._graphs.items() if k[0] == B]
        ms = _time(gr["graph"].replay, 3 * iters)
        out[f"decode {B} at {ctx}"] = {"ms": round(ms, 4), "tokens_per_s": round(B / ms * 1e3)}
        for i in range(B):
            runner.cache.free(i)
    return out


def kernels(s, T: int = 8192, B: int = 64, ctx: int = 4000, iters: int = 10) -> dict:
    """Kernel -> {ms, fraction of the roofline, the like kernel of the Llama-style model and its fraction}."""
    hbm, flops = _peaks()
    d, H, G, dk, E, k, ff = (s[x] for x in ("d", "H", "G", "dk", "E", "top", "ff"))
    F = (k + 1) * ff
    bf, f32 = torch.bfloat16, torch.float32
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    rnd = lambda *sh, dtype=bf: torch.randn(*sh, device="cuda", dtype=f32).mul_(0.5).to(dtype)
    rule = ScoreRule(30.0, distance_slopes(H, "cuda"), CHUNK)
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

    # ---- attention: 4096 tokens of one prompt (one chunk), B decoded rows
    L = CHUNK
    q, kk, vv, gate = rnd(1, L, H, dk), rnd(1, L, G, dk), rnd(1, L, G, dk), rnd(L, H * dk)
    o = torch.empty_like(q)
    roof = 2.0 * H * L * (L + 1) * dk / flops
    row(f"prompt attention {L}", lambda: attn_ops.prompt_attention(q, kk, vv, scale, o, rule, gate), roof,
        ("flash forward", lambda: attn_ops.attention_forward(q, kk, vv, True, scale, out=o, want_lse=False), roof))
    nb = B * (ctx + 15) // 16 + B
    kc, vc = rnd(nb, 16, G, dk), rnd(nb, 16, G, dk)
    per = (ctx + 15) // 16
    bt = torch.randperm(nb, device="cuda")[:B * per].view(B, per).to(torch.int32)
    ctxs = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
    qd, gd, od = rnd(B, H * dk), rnd(B, H * dk), torch.empty(B, H * dk, dtype=bf, device="cuda")
    roof = 4.0 * B * ctx * G * dk / hbm
    row(f"decode attention {B} at {ctx}", lambda: paged_ops.paged_attention_decode(qd, kc, vc, bt, ctxs, scale, od, rule, gd), roof,
        ("paged decode", lambda: paged_ops.paged_attention_decode(qd, kc, vc, bt, ctxs, scale, od), roof))

    # ---- per-head work and norms, prompt and decode sizes
    qg = rnd(dk)
    for t in (T, B):
        z, qkv = rnd(t, 2 * H * dk + 2 * G * dk), rnd(t, (H + 2 * G) * dk)
        slots, pos = torch.randperm(nb * 16, device="cuda")[:t], torch.arange(t, device="cuda")
        vf, mix = rnd(t, G * dk), torch.full((1,), 0.4, device="cuda")

        def like():
            rope_ops.rope_(qkv, H + G, dk, positions=pos)
            paged_ops.kv_append(qkv[:, H * dk:(H + G) * dk], qkv[:, (H + G) * dk:], kc, vc, slots)
        row(f"head norm + mix + append {t}", lambda: head_prep_(z, H, G, dk, dk, q_gamma=qg, k_gamma=qg, v_first=vf, mix=mix, k_cache=kc,
                                                               v_cache=vc, slots=slots), 2.0 * t * dk * (2 * H + 3 * G + 4 * G) / hbm,
            ("rope + append", like, 2.0 * t * dk * (2 * H + 2 * G + 4 * G) / hbm))
        y, x, h, w = rnd(t, d, dtype=f32), rnd(t, d, dtype=f32), rnd(t, d), rnd(d)
        nl = ("rms norm", lambda: norm_ops.norm_forward(h, w, None, 1e-5, True, want_stats=False), 4.0 * t * d / hbm)
        row(f"norm + residual {t}", lambda: norm_ops.residual_norm(y, w, w, 1e-5, x=x, h=h), 14.0 * t * d / hbm, nl)

        # ---- routed feed-forward
        logits = rnd(t, E, dtype=f32)
        idx, rw = moe_ops.route_groups(logits, k, 4, 2)
        row(f"router choice {t}", lambda: moe_ops.route_groups(logits, k, 4, 2), 4.0 * t * (E + 2 * k) / hbm,
            ("moe_route", lambda: moe_ops.route(logits, k), 4.0 * t * (2 * E + 2 * k) / hbm))
        row(f"expert plan {t}", lambda: moe_ops.plan(idx, E), 16.0 * t * k / hbm)
        pl = moe_ops.plan(idx, E)
        row(f"expert scatter {t}", lambda: moe_ops.scatter_tokens(h, pl), 2.0 * t * d * (1 + k) / hbm, nl)
        w1, w2 = rnd(E, 2 * ff, d), rnd(E, d, ff)
        wd1, wd2 = rnd(2 * F, d), rnd(d, F)
        xp = moe_ops.scatter_tokens(h, pl)
        used = int((pl.counts > 0).sum())
        roof = max(4.0 * t * k * d * ff / flops, (4.0 * used * ff * d + 2.0 * t * k * (d + 2 * ff)) / hbm)
        lroof = max(4.0 * t * d * F / flops, (4.0 * F * d + 2.0 * t * (d + 2 * F)) / hbm)
        row(f"experts gate + up {t}", lambda: moe_ops.grouped_gemm(xp, w1, pl), roof, ("dense gate + up", lambda: gemm(h, wd1), lroof))
        gu, gud = moe_ops.grouped_gemm(xp, w1, pl), gemm(h, wd1)
        row(f"expert swiglu {t}", lambda: moe_ops.swiglu_rows(gu, pl), 6.0 * t * k * ff / hbm,
            ("swiglu", lambda: rope_ops.swiglu_forward(gud), 6.0 * t * F / hbm))
        hh, hd = moe_ops.swiglu_rows(gu, pl), rope_ops.swiglu_forward(gud)
        roof = max(2.0 * t * k * d * ff / flops, (2.0 * used * ff * d + 2.0 * t * k * (d + ff)) / hbm)
        lroof = max(2.0 * t * d * F / flops, (2.0 * F * d + 2.0 * t * (d + F)) / hbm)
        row(f"experts down {t}", lambda: moe_ops.grouped_gemm(hh, w2, pl), roof, ("dense down", lambda: gemm(hd, wd2), lroof))
        yp = moe_ops.grouped_gemm(hh, w2, pl)
        row(f"combine + norm + residual {t}", lambda: norm_ops.residual_norm(yp, w, w, 1e-5, x=x, h=h, routed=(pl.slot_pos, rw), add=h),
            t * d * (2.0 * k + 12) / hbm, nl)
        del w1, w2, wd1, wd2, gu, gud, hh, hd, yp, xp
    lg = rnd(B, s["vocab"], dtype=f32)
    row(f"logit cap {B}", lambda: ops.scale_softcap_(lg, 1.0, 30.0), 8.0 * lg.numel() / hbm)
    return out


def run(sizes=None, with_kernels: bool = True) -> dict:
    out = {"metric": "decoder_serving", "dtype": "bf16", "data": "synthetic: random weights and token ids",
           "l2": "kernels: flushed before every launch (256 MiB write); model steps: weights and cache exceed L2", "sizes": {}}
    for name in sizes or SIZES:
        s = SIZES[name]
        e = {"config": {**s, "chunk": CHUNK, "dense_ff": (s["top"] + 1) * s["ff"]}}
        for model, cfg in (("dolurax", _layered(s)), ("llama", _llama(s))):
            e[model] = throughput(cfg)
            torch.cuda.empty_cache()
        if with_kernels:
            e["kernels"] = kernels(s)
            torch.cuda.empty_cache()
        out["sizes"][name] = e
    return out
