"""Plain, slow restatement of the hybrid decoder (Vafodra): one function per mechanism, one sequence at a time, recurrences as
loops over tokens.  Nothing here comes from the product path; the tests compare the framework with it.

All math runs in the dtype of the weights handed in (float32 or float64).
"""
import math

import torch


def dynamic_tanh(x, alpha, weight, bias):
    """A "norm" without statistics: every element is squashed by itself."""
    return torch.tanh(alpha * x) * weight + bias


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def visible(i, j, window, keep):
    """Causal, and (with a window) among the last `window` positions or among the sequence's first `keep`."""
    return j <= i and (not window or i - j < window or j < keep)


def attention(q, k, v, scale, window=0, keep=0, sink=True):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv].  `sink`: a further score 0 without a value takes part in the softmax."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    pos = torch.arange(T)
    see = pos[None, :] <= pos[:, None]
    if window:
        see = see & ((pos[:, None] - pos[None, :] < window) | (pos[None, :] < keep))
    out = torch.empty((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = q[:, h] @ k[:, h // per].T * scale
        s = torch.where(see, s, torch.full_like(s, -math.inf))
        top = s.max(-1, keepdim=True).values
        if sink:
            top = top.clamp(min=0)
        e = torch.exp(s - top)
        den = e.sum(-1, keepdim=True)
        if sink:
            den = den + torch.exp(-top)
        out[:, h] = e / den @ v[:, h // per]
    return out


def windowed_attention(x, w, p, m):
    T = x.shape[0]
    H, G = m["heads"], m["kv_heads"]
    mask = m.get("mask") or {}
    q = (x @ w[p + "q"].T).view(T, H, m["dim"])
    k = (x @ w[p + "k"].T).view(T, G, m["dim"])
    v = (x @ w[p + "v"].T).view(T, G, m["vdim"])
    a = attention(q, k, v, m["scale"], mask.get("size", 0), mask.get("keep_first", 0))
    gate = sigmoid(x @ w[p + "g"].T)                           # one number per head
    return (a * gate[:, :, None]).reshape(T, -1) @ w[p + "o"].T


def causal_conv(x, taps, bias=None):
    """x [T, C], taps [C, n]: the last column of `taps` meets the current token, zeros stand before the first one."""
    T, C = x.shape
    n = taps.shape[1]
    y = torch.zeros_like(x) if bias is None else bias.expand(T, C).clone()
    for t in range(T):
        for i in range(n):
            at = t - (n - 1) + i
            if at >= 0:
                y[t] = y[t] + taps[:, i] * x[at]
    return y


def state_space(x, B, C, dt, a_log, D):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (positive): S <- exp(-exp(a_log) dt) S + dt B x^T, y = S^T C + D x."""
    T, H, P = x.shape
    per = H // B.shape[1]
    y = torch.empty_like(x)
    for h in range(H):
        S = torch.zeros((B.shape[2], P), dtype=x.dtype)
        for t in range(T):
            S = torch.exp(-torch.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * torch.outer(B[t, h // per], x[t, h])
            y[t, h] = S.T @ C[t, h // per] + D[h] * x[t, h]
    return y


def gated_group_norm(y, z, weight, groups, eps):
    """The gate silu(z) comes first; then every one of `groups` equal parts is divided by its own root mean square."""
    T, n = y.shape
    u = (y * silu(z)).view(T, groups, n // groups)
    u = u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps)
    return u.reshape(T, n) * weight


def state_space_mixer(x, w, p, m, eps):
    T = x.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(x @ w[p + "in"].T, [inner, inner + 2 * G * N, H], -1)
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    xs, B, C = torch.split(xbc, [inner, G * N, G * N], -1)
    dt = softplus(dt + w[p + "dt_bias"])
    y = state_space(xs.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), dt, w[p + "A_log"], w[p + "D"])
    return gated_group_norm(y.reshape(T, inner), z, w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


def parallel_mixer(x, w, p, m, eps):
    left = windowed_attention(x, w, p + "left.", m["left"])
    right = state_space_mixer(x, w, p + "right.", m["right"], eps)
    return 0.5 * (rms_norm(left, w[p + "left.out"], eps) + rms_norm(right, w[p + "right.out"], eps))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def gated_delta(q, k, v, beta, decay):
    """q and k [T, G, dk] (ready), v [T, H, dv], beta and decay [T, H]: the state is decayed, corrected towards v at k, then
    read at q."""
    T, H, dv = v.shape
    per = H // k.shape[1]
    o = torch.empty_like(v)
    for h in range(H):
        g = h // per
        S = torch.zeros((k.shape[2], dv), dtype=v.dtype)
        for t in range(T):
            S = decay[t, h] * S
            S = S + torch.outer(k[t, g], beta[t, h] * (v[t, h] - S.T @ k[t, g]))
            o[t, h] = S.T @ q[t, g]
    return o


def delta_mixer(x, w, p, m, eps):
    T = x.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(x @ w[p + c].T, w[p + c + ".conv"])) for c in "qkv")
    q = unit(q.view(T, G, dk)) * dk ** -0.5
    k = unit(k.view(T, G, dk))
    beta = sigmoid(x @ w[p + "b"].T)
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(x @ w[p + "a"].T + w[p + "dt_bias"]))
    o = gated_delta(q, k, v.view(T, H, dv), beta, decay)
    o = rms_norm(o, w[p + "norm"], eps) * silu(x @ w[p + "g"].T).view(T, H, dv)
    return o.reshape(T, -1) @ w[p + "o"].T


def ffn(x, w, p):
    return (torch.relu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None and cfg["layers"][i]["weights_of"] != i:
        i = cfg["layers"][i]["weights_of"]
    return i


def norm(x, w, name):
    return dynamic_tanh(x, w[name + ".alpha"], w[name], w[name + ".b"])


def forward(cfg, w, tokens, trace=None):
    """Logits [T, vocab] of a whole sequence.  `trace`: list that receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}."
        h = norm(x, w, p + "norm1")
        y = {"parallel": parallel_mixer, "delta": delta_mixer}[layer["type"]](h, w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            y = y + ffn(h, w, p + "mlp.")
        x = x + cfg["residual_mult"] * y
        if trace is not None:
            trace.append(x)
    return norm(x, w, "final.norm") @ w["head"].T


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
