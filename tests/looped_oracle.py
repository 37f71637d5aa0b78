"""Plain, slow restatement of the looped decoder (Bikilix): one function per mechanism, one sequence at a time, every token's
experts one by one.  Nothing here comes from the product path; the tests compare the framework with it.

All math runs in the dtype of the weights handed in (float32 or float64).
"""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    """Weight as stored: the scale itself."""
    return unit_rms(x, eps) * w


def centred_norm(x, w, eps):
    """Weight stored as the difference from one."""
    return unit_rms(x, eps) * (1 + w)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def frequencies(rot):
    """(angle per position of every pair, factor on cos and sin)."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def dim_of(turns):                            # the dimension that turns this often over the original context
        return n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(dim_of(s["fast"])), 0)
    hi = min(math.ceil(dim_of(s["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * r + fi * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T, heads, size]: pairs (2i, 2i + 1) of the first rot["dims"] numbers of every head turn with the position."""
    f, m = frequencies(rot)
    y = x.clone()
    for i, fi in enumerate(f):
        a = positions.double() * fi
        c, s = (torch.cos(a) * m).to(x.dtype)[:, None], (torch.sin(a) * m).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i], y[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def softmax_rows(s):
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def attend(q, k, v, scale, window=0):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv]; `window`: how many positions a row sees, itself included (0: all earlier)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    see = back >= 0
    if window:
        see = see & (back < window)
    out = torch.empty((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = q[:, h] @ k[:, h // per].T * scale
        out[:, h] = softmax_rows(s.masked_fill(~see, -math.inf)) @ v[:, h // per]
    return out


def windowed_attention(x, w, p, m):
    T = x.shape[0]
    H, G = m["heads"], m["kv_heads"]
    pos = torch.arange(T)
    q, k, v = (x @ w[p + c].T + w[p + c + ".b"] for c in "qkv")
    q = rotate(q.view(T, H, m["dim"]), pos, m["rot"])
    k = rotate(k.view(T, G, m["dim"]), pos, m["rot"])
    o = attend(q, k, v.view(T, G, m["vdim"]), m["scale"], (m.get("mask") or {}).get("size", 0))
    return o.reshape(T, -1) @ w[p + "o"].T


def latent_attention(x, w, p, m, eps):
    T = x.shape[0]
    H, dn, dr, r = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (rms_norm(x @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).view(T, H, dn + dr)
    joint = x @ w[p + "dkv"].T
    c = rms_norm(joint[:, :r], w[p + "dkv.norm"], eps)
    kr = rotate(joint[:, None, r:], pos, m["rot"])
    q = torch.cat([q[..., :dn], rotate(q[..., dn:], pos, m["rot"])], -1)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, dn), kr.expand(T, H, dr)], -1)
    v = (c @ w[p + "uv"].T).view(T, H, m["vdim"])
    o = attend(q, k, v, m["scale"]).reshape(T, -1)
    return (o * sigmoid(x @ w[p + "g"].T)) @ w[p + "o"].T


def relu2_ff(x, w, p):
    return torch.relu(x @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def clamped_expert(x, w, p, limit):
    g = torch.clamp(x @ w[p + "gate"].T, max=limit)
    u = torch.clamp(x @ w[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def choose(z, correction, top, groups=1, keep=1):
    """One token's experts: (indices, weights) from router logits z [E]."""
    s = sigmoid(z)
    c = s + correction
    per = z.numel() // groups
    if keep < groups:
        rank = [float(torch.sort(c[g * per:(g + 1) * per], descending=True).values[:2].sum()) for g in range(groups)]
        best = sorted(range(groups), key=lambda g: -rank[g])[:keep]
        c = torch.tensor([float(c[e]) if e // per in best else -math.inf for e in range(z.numel())], dtype=torch.float64)
    idx = sorted(range(z.numel()), key=lambda e: -float(c[e]))[:top]
    return idx, s[idx]


def routed_ff(x, w, p, f):
    r = f["router"]
    g = r.get("groups") or {}
    z = x @ w[p + "router"].T
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        idx, ws = choose(z[t], w[p + "correction"], r["top"], g.get("count", 1), g.get("keep", 1))
        for e, we in zip(idx, ws):
            out[t] += we * clamped_expert(x[t], w, f"{p}e{e}.", f["expert"]["limit"])
    return out


def layer(x, w, i, e, eps):
    p = f"l{i}."
    h = centred_norm(x, w[p + "norm1"], eps)
    if e["type"] == "latent_attention":
        y = latent_attention(h, w, p + "mix.", e["mixer"], eps)
    else:
        y = windowed_attention(h, w, p + "mix.", e["mixer"])
    x = x + centred_norm(y, w[p + "norm1b"], eps)
    f = e.get("mlp")
    if f is not None:
        h = centred_norm(x, w[p + "norm2"], eps)
        y = relu2_ff(h, w, p + "mlp.") if f["kind"] == "dense" else routed_ff(h, w, p + "mlp.", f)
        x = x + centred_norm(y, w[p + "norm2b"], eps)
    return x


def order(cfg):
    """Layers in the order they run: (layer, number of the pass that starts in front of it or None)."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    lo, hi = loop["start"], loop["stop"]
    out = [(i, None) for i in range(lo)]
    for t in range(loop["times"]):
        out += [(i, t if i == lo else None) for i in range(lo, hi)]
    return out + [(i, None) for i in range(hi, n)]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; `layers_out` (a list) receives the residual after every layer that runs."""
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    x = x0
    for i, t in order(cfg):
        if t is not None:
            x = torch.cat([x, x0], -1) @ w["loop.in"].T + w["loop.step"][t]
        x = layer(x, w, i, cfg["layers"][i], eps)
        if layers_out is not None:
            layers_out.append(x)
    return centred_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
