"""Checks of the pre-norm decoder (Seredra) that run on any device: each compares the framework with tests/prenorm_oracle.py."""
import torch

import prenorm_oracle as O
from hybrid_checks import poison
from layered_checks import assert_logits, feed, standout_case, tokens
from rustral_b200.models.layered import LayeredConfig
from rustral_b200.serve import ModelRunner
from rustral_b200.serve.weights import InferenceWeights

__all__ = ["assert_logits", "feed", "poison", "standout_case", "tokens"]


def rot(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def att(heads, kv, dim, vdim, conv=4, temp=None, scale=None, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 1.4 * dim ** -0.5, "conv": conv}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mlp": mlp, "mixer": m}


def par(heads, kv, dim, turn, right, scales=(1.3, 0.7), cap=0.0, scale=None, mlp=None):
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale or 1.4 * dim ** -0.5, "rot": turn}
    if cap:
        left["softcap"] = cap
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "right": dict(zip(("inner", "state", "dt_rank", "conv"), right)), "left_scale": scales[0],
                                                      "right_scale": scales[1]}}


def ret(heads, dim, vdim, decay, turn, mlp=None):
    return {"type": "retention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": turn}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def model(layers, width=64, vocab=150, eps=1e-5, scale=2.5):
    return {"architecture": "Seredra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


CONFIGS = {
    # every layer has sizes of its own; two layers use the keys and values of another, one lies between them and it; one layer has no
    # feed-forward; rotated parts that are a piece of a head, all of it, and one pair; with and without cap, temperature and scaling
    "varied": model([par(4, 2, 24, rot(16, 5e3, (4.0, 16, 8.0, 0.5)), (40, 12, 6, 4), cap=4.0, mlp=moe(24, 8, 2)), att(6, 2, 16, 40, 3, (0.6, 7), mlp=dense(56)),
                     ret(3, 16, 24, (0.8, 0.97, 0.999), rot(16, 300.0), mlp=moe(20, 9, 3)), att(4, 2, 16, 40, 2, kv_from=1), ret(2, 32, 16, (1.0, 0.5), rot(8, 1e5), mlp=dense(40)),
                     par(3, 1, 40, rot(2, 50.0), (72, 5, 9, 3), (0.4, 1.9), mlp=moe(16, 5, 5)), att(2, 2, 16, 40, 5, (1.5, 20), kv_from=1, mlp=moe(24, 6, 1))], eps=1e-3),
    # one head, one tap, one state number, one rank, one expert; a coarse eps
    "single": model([att(1, 1, 32, 8, 1, (0.3, 1), mlp=moe(16, 6, 1)), par(1, 1, 8, rot(8, 100.0), (8, 1, 1, 2), (1.0, 1.0), cap=1.5, mlp=moe(20, 1, 1)),
                     ret(1, 8, 16, (0.9,), rot(4, 1e4), mlp=dense(24)), att(1, 1, 32, 8, 2, kv_from=0)], eps=1e-2, scale=1.0),
    # sizes as large as the kernels' tiles or larger, and no multiples of them
    "wide": model([par(8, 2, 128, rot(128, 5e4, (6.0, 40, 6.0, 0.25)), (200, 40, 24, 4), cap=12.0, mlp=dense(96)), att(6, 3, 104, 72, 4, (0.5, 33), mlp=moe(40, 16, 4)),
                   ret(4, 64, 128, (0.9, 0.98, 0.996, 0.9995), rot(64, 1e4), mlp=moe(32, 8, 2)), att(12, 3, 104, 72, 3, (0.25, 64), kv_from=1, mlp=dense(96)),
                   par(4, 4, 64, rot(32, 1e4), (128, 16, 16, 4), (0.9, 1.2), mlp=None)], width=128, vocab=260),
    # the same without routed experts
    "dense": model([par(8, 2, 128, rot(128, 5e4, (6.0, 40, 6.0, 0.25)), (200, 40, 24, 4), cap=12.0, mlp=dense(96)), att(6, 3, 104, 72, 4, (0.5, 33), mlp=dense(40)),
                    ret(4, 64, 128, (0.9, 0.98, 0.996, 0.9995), rot(64, 1e4), mlp=dense(72)), att(12, 3, 104, 72, 3, (0.25, 64), kv_from=1),
                    par(4, 4, 64, rot(32, 1e4), (128, 16, 16, 4), (0.9, 1.2), mlp=None)], width=136, vocab=260),
    # sizes that are no multiple of 8, rotated parts of odd width
    "odd": model([par(6, 3, 20, rot(6, 4e3, (3.0, 30, 8.0, 0.5)), (36, 7, 5, 4), cap=6.0, mlp=dense(44)), ret(3, 12, 10, (0.7, 0.95, 0.99), rot(10, 500.0), mlp=moe(20, 10, 3)),
                  att(6, 3, 13, 11, 4, (0.8, 11), mlp=dense(50)), att(3, 3, 13, 11, 4, kv_from=2), par(2, 1, 14, rot(14, 60.0), (27, 3, 4, 2))], width=72),
    # heads and states too large for the tensor-core kernels
    "large": model([par(2, 1, 136, rot(136, 1e3), (24, 72, 8, 4), cap=8.0, mlp=dense(64)), ret(1, 144, 40, (0.99,), rot(144, 1e4), mlp=moe(16, 4, 2)),
                    att(2, 1, 160, 144, 4, (0.5, 16), mlp=dense(32)), par(1, 1, 32, rot(16, 1e3), (16, 200, 3, 4))]),
}


def weights(cfg, seed=0):
    """Random checkpoint, rounded to bf16; nothing is 0 or 1 that could be left out unnoticed."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in LayeredConfig.from_json(cfg).tensor_shapes().items():
        t = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if last.startswith("norm"):
            t = (1.6 if ".mix." in name else 1.0) + 0.3 * t                      # scores that stand out
        elif name.endswith(".dt.b"):
            t = 1.0 * t - 2.5
        elif last == "b":
            t = 0.3 * t
        elif last == "r1":
            t = 0.2 + t.abs()
        elif last == "r2":
            t = 0.05 + 0.4 * t.abs()
        elif last == "A_log":
            t = 1.2 * t - 0.5
        elif last == "D":
            t = 1.0 + 0.3 * t
        elif last == "conv":
            t = t * shape[-1] ** -0.5
        elif last == "embed":
            t = 0.4 * t
        else:
            t = t * shape[-1] ** -0.5 * (2.5 if last in ("router", "gate") else 1.0)
        w[name] = t.bfloat16()
    return w


def runner(cfg, w, device="cpu", dtype=torch.float32, blocks=64, block_size=16, graphs=True, slots=4):
    lc = LayeredConfig.from_json(cfg)
    r = ModelRunner(lc, params=InferenceWeights.layered(lc, device, dtype, w), device=device, num_blocks=blocks, block_size=block_size, num_slots=slots)
    r.use_graphs = graphs
    return r


def reference(cfg, w, toks):
    return O.forward(cfg, {k: v.double() for k, v in w.items()}, toks).float()


def sequence(cfg, w, n, seed=1, dtype=torch.float32, gap=0.03):
    """Random tokens.  For a comparison in bf16 the ones with a close call are replaced (one expert's logit near another's at the edge of
    the choice): rounding would change which experts are chosen, and with it the state and keys that all later tokens see."""
    toks = tokens(cfg, n, seed)
    if dtype == torch.float32:
        return toks
    g, plain, wd = torch.Generator().manual_seed(1000 + seed), O.choose, {k: v.double() for k, v in w.items()}
    calls = []

    def recorded(z, top):
        v = torch.sort(z, descending=True).values
        calls.append(1.0 if top == z.numel() else float((v[top - 1] - v[top]) / z.pow(2).mean().sqrt()))
        return plain(z, top)
    try:
        O.choose = recorded
        for _ in range(400):
            calls.clear()
            O.forward(cfg, wd, toks)
            if not calls:
                return toks
            tight = (torch.tensor(calls).view(-1, n).amin(0) < gap).nonzero()
            if not len(tight):
                return toks
            for i in tight[:, 0].tolist():
                toks[i] = int(torch.randint(0, cfg["vocab"], (1,), generator=g))
    finally:
        O.choose = plain
    raise RuntimeError("no sequence without close calls found")


def check_prefill_portions_and_decode(name, device, dtype, n=90, plans=None):
    cfg = CONFIGS[name]
    w = weights(cfg, 0)
    toks = sequence(cfg, w, n, 1, dtype)
    want = reference(cfg, w, toks)
    r = runner(cfg, w, device, dtype)
    plans = plans or {"whole": [], "decoded": list(range(1, n)), "pairs": list(range(2, n, 2)), "threes": list(range(3, n, 3)), "prompt then decode": list(range(41, n)),
                      "page edges": [15, 16, 17, 31, 33, 48, 64, 66], "temperature edges": [6, 7, 13, 14, 18, 19, 20, 32, 33, 38, 39], "two after one": [1, 3, 5, 6, 8]}
    for seq, (what, cuts) in enumerate(plans.items()):
        poison(r)
        assert_logits(feed(r, seq, toks, [c for c in cuts if c < n]), want, dtype, (name, what))
        r.cache.free(seq)                               # the next plan uses the same pages and slots, in another order
        r.cache.allocate(1000 + seq, 16 * (1 + seq % 3))
        if seq % 2:
            r.cache.free(1000 + seq - 1)
            r.cache.free(1000 + seq)


def check_mixed_batch_with_reused_pages(name, device, dtype):
    cfg = CONFIGS[name]
    w = weights(cfg, 3)
    lens = [50, 9, 33, 70, 2, 41]
    toks = [sequence(cfg, w, n, 10 + i, dtype) for i, n in enumerate(lens)]
    want = [reference(cfg, w, t) for t in toks]
    r = runner(cfg, w, device, dtype, blocks=11, slots=3)        # far fewer pages and slots than all requests hold together
    poison(r)
    portions = [13, 2, 1, 7, 1, 1, 20, 3]
    live, waiting, got, step = {}, list(range(len(lens))), {i: [] for i in range(len(lens))}, 0
    while live or waiting:
        while waiting and len(live) < 3 and sum(-(-lens[i] // 16) for i in [*live, waiting[0]]) <= 11:
            live[waiting.pop(0)] = 0
        chunks, dec = [], []
        for k, (i, at) in enumerate(list(live.items())):
            if (step + k) % 5 == 4:
                continue                                 # left out of this step
            n = min(portions[(step + 3 * k) % len(portions)], lens[i] - at)
            assert r.cache.allocate(i, at + n)
            if n == 1 and at > 0:
                dec.append((i, toks[i][at], at + 1))
            else:
                chunks.append((i, toks[i][at:at + n], at, list(range(n))))
            live[i] = at + n
        if chunks or dec:
            a, b = r.step(chunks, [d[0] for d in dec], [d[1] for d in dec], [d[2] for d in dec])
            for c, lg in zip(chunks, a):
                got[c[0]].append(lg.float().cpu())
            for j, d in enumerate(dec):
                got[d[0]].append(b[j:j + 1].float().cpu())
        for i in [i for i, at in live.items() if at == lens[i]]:
            r.cache.free(i)
            del live[i]
        step += 1
    for i in range(len(lens)):
        assert_logits(torch.cat(got[i]), want[i], dtype, (name, "request", i))
    assert r.cache.free_blocks == 11 and r.cache.free_slots == 3


def check_long_decoding(name, device, dtype, n=200):
    cfg = CONFIGS[name]
    w = weights(cfg, 5)
    toks = sequence(cfg, w, n, 4, dtype)
    got = feed(runner(cfg, w, device, dtype), 0, toks, list(range(3, n)))
    assert_logits(got, reference(cfg, w, toks), dtype, (name, "long decoding"))
