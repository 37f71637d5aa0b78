"""Checks of the layered decoder that run on any device: each compares the framework with tests/layered_oracle.py."""
import torch

import layered_oracle as O
from rustral_b200.models.layered import LayeredConfig
from rustral_b200.serve import ModelRunner
from rustral_b200.serve.weights import InferenceWeights


def _layer(heads, kv, dim, vdim, chunk=0, cap=0.0, v_mix=True, mlp=True, scale=None, experts=8, top=2, groups=(4, 2), ff=24,
           shared=40):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "v_mix": v_mix}
    if chunk:
        m["mask"] = {"size": chunk}
    if cap:
        m["softcap"] = cap
    f = None
    if mlp:
        f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
        if groups:
            f["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
        if shared:
            f["shared"] = {"ff": shared}
    return {"type": "attention", "mixer": m, "mlp": f}


def _model(layers, width=64, vocab=150, eps=1e-5, scale=1.5, cap=12.0):
    return {"architecture": "Dolurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": scale,
            "logit_softcap": cap, "layers": layers}


CONFIGS = {
    # every layer differs; the first layer does not mix values, one layer has no feed-forward
    "varied": _model([_layer(4, 2, 24, 16, chunk=20, cap=9.0, v_mix=False), _layer(6, 2, 40, 16, chunk=33, cap=14.0),
                      _layer(4, 2, 16, 16, chunk=7, mlp=False), _layer(2, 2, 64, 16, cap=6.0, groups=None, top=3, shared=0)]),
    # one head, one expert chosen, no cap, no groups of more than one expert kept, no output cap, a coarse eps
    "single": _model([_layer(1, 1, 32, 32, chunk=16, top=1, groups=(8, 1), ff=20), _layer(1, 1, 32, 32, chunk=1, experts=1, top=1,
                                                                                         groups=None)], eps=1e-2, cap=None),
    # wider heads and chunks that are no multiple of a page or a tile
    "wide": _model([_layer(8, 2, 128, 72, chunk=150, cap=20.0, experts=16, top=4, groups=(4, 3)),
                    _layer(8, 2, 96, 72, chunk=150, cap=20.0, experts=16, top=4, groups=(2, 1))], width=128, vocab=260),
    # head sizes that are no multiple of 8, several heads per group
    "odd": _model([_layer(6, 3, 20, 12, chunk=24, cap=10.0), _layer(6, 3, 20, 12, chunk=24, cap=10.0)], width=72),
}


def weights(cfg, seed=0):
    """Random checkpoint, rounded to bf16; norms, mixing shares and biases are not 1, 0.5 or 0."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in LayeredConfig.from_json(cfg).tensor_shapes().items():
        t = torch.randn(shape, generator=g)
        if name.endswith(".b"):
            t = 0.2 * t
        elif "norm" in name:
            t = 1.0 + 0.3 * t
        elif name.endswith("vmix"):
            t = torch.sigmoid(t)
        elif name.endswith("router"):
            t = t * 0.4
        elif name != "embed":
            t = t * shape[-1] ** -0.5
        if name.endswith((".q.norm", ".k.norm")):
            t = t * 1.6                                  # scores that stand out
        w[name] = t.bfloat16()
    return w


def runner(cfg, w, device="cpu", dtype=torch.float32, blocks=64, block_size=16, graphs=True):
    lc = LayeredConfig.from_json(cfg)
    r = ModelRunner(lc, params=InferenceWeights.layered(lc, device, dtype, w), device=device, num_blocks=blocks, block_size=block_size)
    r.use_graphs = graphs
    return r


def reference(cfg, w, tokens):
    return O.forward(cfg, {k: v.double() for k, v in w.items()}, tokens).float()


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def assert_logits(got, want, dtype, what=""):
    """Per position: rms difference over rms of the reference.  In bf16 one position in ten may be off by more (a routing
    score near another's)."""
    got = got[:, :want.shape[1]].float().cpu()
    d = got - want
    err = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
    assert torch.isfinite(err).all(), what
    if dtype == torch.float32:
        assert err.max() < 2e-4, (what, float(err.max()), int(err.argmax()))
    else:
        bad = (err > 0.05).float().mean()
        assert bad <= 0.1 and err.median() < 0.03, (what, float(err.max()), int(err.argmax()), float(bad), float(err.median()))


def feed(r, seq, toks, cuts):
    """Runs `toks` of sequence `seq` in portions ending at `cuts`; single tokens after the first go through decode."""
    out, lo = [], 0
    for hi in [*cuts, len(toks)]:
        if hi <= lo:
            continue
        assert r.cache.allocate(seq, hi)
        if hi - lo == 1 and lo > 0:
            out.append(r.step([], [seq], [toks[lo]], [hi])[1].clone())
        else:
            out.append(r.step([(seq, toks[lo:hi], lo, list(range(hi - lo)))], [], [], [])[0][0].clone())
        lo = hi
    return torch.cat(out)


def check_prefill_portions_and_decode(name, device, dtype, n=90):
    cfg = CONFIGS[name]
    w = weights(cfg)
    toks = tokens(cfg, n)
    want = reference(cfg, w, toks)
    r = runner(cfg, w, device, dtype)
    seq = 0
    plans = {"whole": [], "decoded": list(range(1, n)), "pairs": list(range(2, n, 2)), "prompt then decode": list(range(41, n)),
             "page edges": [15, 16, 17, 31, 33, 48, 64, 66], "chunk edges": [7, 19, 20, 21, 23, 32, 33, 34, 40, 66, 67]}
    for what, cuts in plans.items():
        assert_logits(feed(r, seq, toks, cuts), want, dtype, (name, what))
        r.cache.free(seq)                               # the next plan uses the same pages, in another order
        r.cache.allocate(1000 + seq, 16 * (1 + seq))    # ... from another place on
        r.cache.free(1000 + seq - 1)
        seq += 1


def check_mixed_batch_with_reused_pages(name, device, dtype):
    cfg = CONFIGS[name]
    w = weights(cfg, 3)
    lens = [50, 9, 33, 70, 2, 41]
    toks = [tokens(cfg, n, 10 + i) for i, n in enumerate(lens)]
    want = [reference(cfg, w, t) for t in toks]
    r = runner(cfg, w, device, dtype, blocks=11)         # far fewer pages than all requests hold together
    for c in (r.cache.k, r.cache.v):
        for t in c:
            t.fill_(1e4)                                 # what an earlier owner of the page left
    portions = [13, 2, 1, 7, 1, 1, 20, 3]
    live, waiting, got, step = {}, list(range(len(lens))), {i: [] for i in range(len(lens))}, 0
    while live or waiting:
        while waiting and len(live) < 3 and sum(-(-lens[i] // 16) for i in [*live, waiting[0]]) <= 11:
            live[waiting.pop(0)] = 0
        chunks, dec, order = [], [], []
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
    w = weights(cfg, 5)
    toks = tokens(cfg, n, 4)
    want = reference(cfg, w, toks)
    got = feed(runner(cfg, w, device, dtype), 0, toks, list(range(3, n)))
    assert_logits(got, want, dtype, (name, "long decoding"))


def standout_case(i, j, T, heads, kv, dk, dv, seed=0):
    """q, k, v of T tokens in which query i matches key j far better than any other pair does."""
    g = torch.Generator().manual_seed(seed)
    q, k = torch.randn(T, heads, dk, generator=g), torch.randn(T, kv, dk, generator=g)
    v = torch.randn(T, kv, dv, generator=g)
    u = torch.randn(dk, generator=g)
    u = u / u.norm()
    q[i], k[j] = 6.0 * u, 6.0 * u
    return q.bfloat16().float(), k.bfloat16().float(), v.bfloat16().float()
