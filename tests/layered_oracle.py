"""Plain, slow restatement of the layered decoder (Dolurax): one function per mechanism, one sequence at a time, dense
loops where they are the clearest form.  Nothing here comes from the product path; the tests compare the framework with it.

All math runs in the dtype of the weights handed in (float32 or float64).
"""
import math

import torch


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def layer_norm(x, weight, bias, eps):
    mean = x.mean(-1, keepdim=True)
    dev = x - mean
    return dev / torch.sqrt((dev * dev).mean(-1, keepdim=True) + eps) * weight + bias


def silu(z):
    return z / (1 + torch.exp(-z))


def soft_cap(z, cap):
    return z if not cap else cap * torch.tanh(z / cap)


def head_slopes(heads, dtype=torch.float64):
    """One distance slope per query head: a geometric sequence from 2^(-8/H) down to 2^-8."""
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=dtype)


def visible(i, j, chunk):
    """Causal, and (with a chunk size) in the same chunk of the sequence."""
    return j <= i and (not chunk or i // chunk == j // chunk)


def mix_values(v, v_first, lam):
    return (1 - lam) * v + lam * v_first


def attention(q, k, v, scale, cap, chunk):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv]: scores are scaled, capped, then lowered by slope * distance."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    slopes = head_slopes(H, q.dtype)
    pos = torch.arange(T)
    dist = (pos[:, None] - pos[None, :]).to(q.dtype)
    see = pos[None, :] <= pos[:, None]
    if chunk:
        see = see & (pos[:, None] // chunk == pos[None, :] // chunk)
    out = torch.empty((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        g = h // per
        s = soft_cap(q[:, h] @ k[:, g].T * scale, cap) - slopes[h] * dist
        s = torch.where(see, s, torch.full_like(s, -math.inf))
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = e / e.sum(-1, keepdim=True) @ v[:, g]
    return out


def mixer(x, w, p, m, eps, v_first):
    """The attention sublayer.  `v_first`: the first mixing layer's own values of every token (None before it).  Returns
    (output, the values that the layer attends with before they were mixed)."""
    T = x.shape[0]
    H, G = m["heads"], m["kv_heads"]
    q = rms_norm((x @ w[p + "q"].T).view(T, H, m["dim"]), w[p + "q.norm"], eps)
    k = rms_norm((x @ w[p + "k"].T).view(T, G, m["dim"]), w[p + "k.norm"], eps)
    own = (x @ w[p + "v"].T).view(T, G, m["vdim"])
    v = own
    if m.get("v_mix") and v_first is not None:
        v = mix_values(own, v_first, w[p + "vmix"])
    a = attention(q, k, v, m["scale"], m.get("softcap"), (m.get("mask") or {}).get("size"))
    gate = 1 / (1 + torch.exp(-(x @ w[p + "g"].T)))
    return (a.reshape(T, -1) * gate) @ w[p + "o"].T, own


def gated_ffn(x, w, p):
    return (silu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def choose_experts(scores, top, groups):
    """Indices of the `top` largest scores among the experts of the best groups (a group counts as its best expert)."""
    s = scores.clone()
    if groups:
        n = scores.numel() // groups["count"]
        best = scores.view(groups["count"], n).max(-1).values
        kept = torch.sort(best, descending=True, stable=True).indices[:groups["keep"]].tolist()
        for g in range(groups["count"]):
            if g not in kept:
                s[g * n:(g + 1) * n] = -math.inf
    return torch.sort(s, descending=True, stable=True).indices[:top].tolist()


def moe(x, w, p, m):
    r = m["router"]
    z = x @ w[p + "router"].T
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        idx = choose_experts(s[t], r["top"], r.get("groups"))
        tot = sum(s[t, i] for i in idx) + 1e-20
        for i in idx:
            y[t] += s[t, i] / tot * gated_ffn(x[t], w, f"{p}e{i}.")
    if m.get("shared"):
        y = y + gated_ffn(x, w, p + "shared.")
    return y


def forward(cfg, w, tokens, trace=None):
    """Logits [T, vocab] of a whole sequence.  `trace`: list that receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        m = layer["mixer"]
        y, own = mixer(x, w, p + "mix.", m, eps, v_first)
        if m.get("v_mix") and v_first is None:
            v_first = own
        x = x + layer_norm(y, w[p + "norm1"], w[p + "norm1.b"], eps)
        if layer.get("mlp"):
            x = x + layer_norm(moe(x, w, p + "mlp.", layer["mlp"]), w[p + "norm2"], w[p + "norm2.b"], eps)
        if trace is not None:
            trace.append(x)
    x = layer_norm(x, w["final.norm"], w["final.norm.b"], eps)
    return soft_cap(x @ w["head"].T * cfg.get("logit_scale", 1.0), cfg.get("logit_softcap"))


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
