"""Checks of the hybrid decoder (Vafodra) that run on any device: each compares the framework with tests/hybrid_oracle.py."""
import torch

import hybrid_oracle as O
from layered_checks import assert_logits, feed, standout_case, tokens
from rustral_b200.models.layered import LayeredConfig
from rustral_b200.serve import ModelRunner
from rustral_b200.serve.weights import InferenceWeights

__all__ = ["assert_logits", "feed", "standout_case", "tokens"]


def left(heads, kv, dim, vdim, window, keep, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 1.5 * dim ** -0.5,
            "mask": {"size": window, "keep_first": keep}}


def right(heads, vdim, state, groups, parts, conv):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": parts, "conv": conv}


def par(a, r, ff=None, of=None):
    e = {"type": "parallel", "mixer": {"left": a, "right": r}, "mlp": {"kind": "dense", "ff": ff} if ff else None}
    return e if of is None else {**e, "weights_of": of}


def delta(heads, kv, dim, vdim, conv, ff=None, of=None):
    e = {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv},
         "mlp": {"kind": "dense", "ff": ff} if ff else None}
    return e if of is None else {**e, "weights_of": of}


def model(layers, width=64, vocab=150, eps=1e-5, scale=3.5, mult=0.7):
    return {"architecture": "Vafodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "residual_mult": mult, "layers": layers}


_A = left(4, 2, 24, 16, 20, 3)
_R = right(6, 24, 16, 3, 4, 4)
CONFIGS = {
    # every kind of layer, other sizes on either side, shared tensors (also of a later layer and through another sharer), layers
    # without a feed-forward
    "varied": model([par(_A, _R, 40), delta(6, 3, 16, 24, 3, 56), par(left(6, 3, 40, 24, 7, 9), right(2, 40, 24, 1, 5, 3)),
                     par(_A, _R, 40, of=0), delta(6, 3, 16, 24, 3, 56, of=1), delta(2, 1, 8, 32, 2, of=6), delta(2, 1, 8, 32, 2),
                     par(_A, _R, 40, of=3)], eps=1e-3),
    # one head, one group, windows of one token, no kept tokens, filters of one tap
    "single": model([par(left(1, 1, 32, 32, 1, 0), right(1, 16, 8, 1, 1, 1), 20), delta(1, 1, 8, 8, 1, 24),
                     par(left(1, 1, 16, 8, 16, 0), right(1, 8, 8, 1, 1, 2))], eps=1e-2, scale=1.0, mult=1.0),
    # heads as wide as the kernels' tiles, windows that are no multiple of a page or a tile, several column tiles
    "wide": model([par(left(8, 2, 128, 72, 150, 5), right(4, 72, 128, 2, 2, 4), 96), delta(4, 2, 128, 136, 4, 104),
                   par(left(4, 4, 64, 128, 33, 130), right(2, 128, 64, 1, 4, 4), 96)], width=128, vocab=260),
    # sizes that are no multiple of 8, long filters, kept tokens beyond the window
    "odd": model([par(left(6, 3, 20, 12, 24, 30), right(3, 20, 12, 3, 2, 6), 36), delta(4, 2, 20, 12, 5, 44)], width=70),
}


def weights(cfg, seed=0):
    """Random checkpoint, rounded to bf16; nothing is 0 or 1 that could be left out unnoticed."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in LayeredConfig.from_json(cfg).tensor_shapes().items():
        t = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if last == "alpha":
            t = 0.6 + 0.2 * torch.rand(shape, generator=g)
        elif last == "A_log":
            t = torch.empty(shape).uniform_(-3.0, 1.5, generator=g)
        elif last == "dt_bias":
            t = t * 0.5 - 1.0
        elif last == "b" and len(shape) == 1:
            t = 0.2 * t
        elif last in ("norm", "norm1", "out"):
            t = 1.0 + 0.3 * t
        elif last == "conv":
            t = t * 0.7
        elif last == "embed":
            t = 0.4 * t
        elif last != "D":
            t = t * shape[-1] ** -0.5
        w[name] = t.bfloat16()
    return w


def runner(cfg, w, device="cpu", dtype=torch.float32, blocks=64, block_size=16, graphs=True, slots=8):
    lc = LayeredConfig.from_json(cfg)
    r = ModelRunner(lc, params=InferenceWeights.layered(lc, device, dtype, w), device=device, num_blocks=blocks, block_size=block_size,
                    num_slots=slots)
    r.use_graphs = graphs
    return r


def poison(r):
    """What an earlier owner left in pages and state slots."""
    for c in (r.cache.k, r.cache.v):
        for t in c:
            if t is not None:
                t.fill_(1e4)
    for d in r.cache.state:
        for t in d.values():
            t.fill_(1e4)


def reference(cfg, w, toks):
    return O.forward(cfg, {k: v.double() for k, v in w.items()}, toks).float()


def check_prefill_portions_and_decode(name, device, dtype, n=90, plans=None):
    cfg = CONFIGS[name]
    w = weights(cfg)
    toks = tokens(cfg, n)
    want = reference(cfg, w, toks)
    r = runner(cfg, w, device, dtype)
    plans = plans or {"whole": [], "decoded": list(range(1, n)), "pairs": list(range(2, n, 2)), "prompt then decode": list(range(41, n)),
                      "page edges": [15, 16, 17, 31, 33, 48, 64, 66], "window edges": [3, 4, 7, 19, 20, 21, 23, 24, 25, 63, 65],
                      "two after one": [1, 3, 5, 6, 8]}
    for seq, (what, cuts) in enumerate(plans.items()):
        poison(r)
        assert_logits(feed(r, seq, toks, [c for c in cuts if c < n]), want, dtype, (name, what))
        r.cache.free(seq)                               # the next plan uses the same pages and another slot order
        r.cache.allocate(1000 + seq, 16 * (1 + seq % 3))
        if seq % 2:
            r.cache.free(1000 + seq - 1)


def check_mixed_batch_with_reused_pages_and_slots(name, device, dtype):
    cfg = CONFIGS[name]
    w = weights(cfg, 3)
    lens = [50, 9, 33, 70, 2, 41]
    toks = [tokens(cfg, n, 10 + i) for i, n in enumerate(lens)]
    want = [reference(cfg, w, t) for t in toks]
    r = runner(cfg, w, device, dtype, blocks=11, slots=3)    # far fewer pages and slots than all requests hold together
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
    toks = tokens(cfg, n, 4)
    got = feed(runner(cfg, w, device, dtype), 0, toks, list(range(3, n)))
    assert_logits(got, reference(cfg, w, toks), dtype, (name, "long decoding"))


def oracle_state_space(segs, x, B, C, dt_raw, dt_bias, a_log, D, past):
    """Every segment through the plain recurrence.  `past`: segment -> (x, B, C, dt_raw) rows that came before it."""
    y = torch.empty_like(x)
    for i, (first, n, _, _) in enumerate(segs):
        rows = slice(first, first + n)
        parts = [t[rows] for t in (x, B, C, dt_raw)]
        if i in past:
            parts = [torch.cat([p, t]) for p, t in zip(past[i], parts)]
        o = O.state_space(parts[0], parts[1], parts[2], O.softplus(parts[3] + dt_bias), a_log, D)
        y[rows] = o[-n:]
    return y
