"""Checks of the looped decoder (Bikilix) that run on any device: each compares the framework with tests/looped_oracle.py."""
import torch

import looped_oracle as O
from layered_checks import assert_logits, feed, standout_case, tokens
from rustral_b200.models.layered import LayeredConfig
from rustral_b200.serve import ModelRunner
from rustral_b200.serve.weights import InferenceWeights

__all__ = ["assert_logits", "feed", "standout_case", "tokens"]


def win(heads, kv, dim, vdim, size, rot, base=5000.0, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 1.7 * dim ** -0.5,
                                                       "mask": {"size": size}, "rot": {"dims": rot, "base": base}}}


def lat(heads, dim, rot, vdim, rank, q_rank, base=8000.0, scaling=(4.0, 16, 8.0, 0.5), scale=None, mlp=None):
    r = {"dims": rot, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank,
                                                              "scale": scale or 1.7 * (dim + rot) ** -0.5, "rot": r}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, groups=None, limit=1.5):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": r}


def model(layers, loop=None, width=64, vocab=150, eps=1e-5, scale=2.5):
    m = {"architecture": "Bikilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    return m if loop is None else {**m, "loop": dict(zip(("start", "stop", "times"), loop))}


CONFIGS = {
    # both mixers and both feed-forwards on either side of and inside the loop, every layer with sizes of its own, one without a
    # feed-forward; rotated parts that are a piece of a head, all of it, and one pair
    "varied": model([win(4, 2, 24, 16, 20, 8, mlp=moe(24, 8, 2, (4, 2))), lat(3, 16, 8, 24, 40, 32, mlp=dense(56)),
                     win(6, 3, 16, 40, 7, 16, mlp=moe(20, 9, 3, (3, 2), 0.7)), lat(5, 24, 16, 8, 24, 48, base=3e5, scaling=(6.0, 40, 6.0, 0.25)),
                     lat(2, 8, 2, 16, 16, 24, scaling=None, mlp=moe(24, 6, 4)), win(2, 2, 32, 24, 33, 2, mlp=dense(40))], (1, 4, 2), eps=1e-3),
    # the whole model is the loop, three passes; one head, windows of one token, one expert of one group
    "single": model([win(1, 1, 32, 32, 1, 4, mlp=moe(16, 6, 1, (6, 1))), lat(1, 8, 8, 8, 8, 8, mlp=moe(20, 1, 1)), win(1, 1, 16, 8, 16, 16, mlp=dense(24))],
                    (0, 3, 3), eps=1e-2, scale=1.0),
    # heads and latents as wide as the kernels' tiles or wider, more heads than one tile takes, windows that are no multiple of a page or
    # a tile; the loop is the last layer
    "wide": model([win(8, 2, 128, 72, 150, 64, mlp=moe(40, 16, 4, (4, 3), 4.0)), lat(20, 128, 64, 128, 136, 72, mlp=dense(96)),
                   win(4, 4, 64, 64, 70, 32, mlp=dense(96)), lat(5, 64, 32, 72, 512, 64, mlp=moe(32, 8, 2))], (3, 4, 4), width=128, vocab=260),
    # sizes that are no multiple of 8, rotated parts of odd width, one pass, no groups
    "odd": model([win(6, 3, 20, 12, 24, 6, mlp=moe(20, 10, 3, (5, 3))), lat(3, 12, 6, 10, 20, 28, mlp=dense(44)), lat(2, 13, 4, 11, 9, 7, mlp=dense(50))],
                 (1, 2, 1), width=72),
    # no loop
    "straight": model([lat(4, 40, 16, 32, 72, 40, mlp=moe(32, 10, 3, (5, 2), 0.8)), win(4, 1, 104, 96, 30, 20, mlp=dense(64))], width=96),
}


def weights(cfg, seed=0, dtype=torch.float32):
    """Random checkpoint, rounded to bf16; nothing is 0 or 1 that could be left out unnoticed, choice corrections have both signs.  For a
    comparison in bf16 the corrections are further apart than scores can be, so that no rounding changes which experts are chosen."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    lc = LayeredConfig.from_json(cfg)
    for name, shape in lc.tensor_shapes().items():
        t = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if last == "correction":
            if dtype == torch.float32:
                t = 0.6 * t - 0.4
            else:                                        # groups apart, and the experts of a group apart
                n = lc.layers[int(name[1:name.index(".")])].mlp.groups
                order = [torch.randperm(n, generator=g), *(torch.randperm(shape[0] // n, generator=g) for _ in range(n))]
                t = 1.25 * (torch.cat([order[0][i] * (shape[0] // n) + order[1 + i] for i in range(n)]) - 0.7 * shape[0])
        elif last.startswith("norm") and name != "final.norm" and ".mix." not in name or name == "final.norm":
            t = 0.3 * t
        elif last == "norm":
            t = 1.0 + 0.3 * t
        elif last in ("b", "step"):
            t = 0.3 * t
        elif last == "embed":
            t = 0.4 * t
        else:
            t = t * shape[-1] ** -0.5 * (2.0 if last in ("router", "gate") else 1.0)
        w[name] = t.bfloat16()
    return w


def runner(cfg, w, device="cpu", dtype=torch.float32, blocks=64, block_size=16, graphs=True):
    lc = LayeredConfig.from_json(cfg)
    r = ModelRunner(lc, params=InferenceWeights.layered(lc, device, dtype, w), device=device, num_blocks=blocks, block_size=block_size)
    r.use_graphs = graphs
    return r


def poison(r):
    """What an earlier owner left in the pages."""
    for c in (r.cache.k, r.cache.v):
        for t in c:
            t.fill_(1e4)


def reference(cfg, w, toks):
    return O.forward(cfg, {k: v.double() for k, v in w.items()}, toks).float()


def check_prefill_portions_and_decode(name, device, dtype, n=90, plans=None):
    cfg = CONFIGS[name]
    w = weights(cfg, 0, dtype)
    toks = tokens(cfg, n)
    want = reference(cfg, w, toks)
    r = runner(cfg, w, device, dtype)
    plans = plans or {"whole": [], "decoded": list(range(1, n)), "pairs": list(range(2, n, 2)), "prompt then decode": list(range(41, n)),
                      "page edges": [15, 16, 17, 31, 33, 48, 64, 66], "window edges": [6, 7, 8, 19, 20, 21, 23, 24, 25, 30, 33, 34],
                      "two after one": [1, 3, 5, 6, 8]}
    for seq, (what, cuts) in enumerate(plans.items()):
        poison(r)
        assert_logits(feed(r, seq, toks, [c for c in cuts if c < n]), want, dtype, (name, what))
        r.cache.free(seq)                               # the next plan uses the same pages, in another order
        r.cache.allocate(1000 + seq, 16 * (1 + seq % 3))
        if seq % 2:
            r.cache.free(1000 + seq - 1)


def check_mixed_batch_with_reused_pages(name, device, dtype):
    cfg = CONFIGS[name]
    w = weights(cfg, 3, dtype)
    lens = [50, 9, 33, 70, 2, 41]
    toks = [tokens(cfg, n, 10 + i) for i, n in enumerate(lens)]
    want = [reference(cfg, w, t) for t in toks]
    r = runner(cfg, w, device, dtype, blocks=11)         # far fewer pages than all requests hold together
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
    assert r.cache.free_blocks == 11


def check_long_decoding(name, device, dtype, n=200):
    cfg = CONFIGS[name]
    w = weights(cfg, 5, dtype)
    toks = tokens(cfg, n, 4)
    got = feed(runner(cfg, w, device, dtype), 0, toks, list(range(3, n)))
    assert_logits(got, reference(cfg, w, toks), dtype, (name, "long decoding"))
