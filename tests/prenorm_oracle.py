"""Plain, slow restatement of the pre-norm decoder (Seredra): one function per mechanism, one sequence at a time, one token at a time where
state is carried.  Nothing here comes from the product path; the tests compare the framework with it.

All math runs in the dtype of the weights handed in (float32 or float64).
"""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))


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
    """x [T, heads, size]: numbers i and i + dims / 2 of every head turn together with the position."""
    f, m = frequencies(rot)
    half = rot["dims"] // 2
    y = x.clone()
    for i, fi in enumerate(f):
        a = positions.double() * fi
        c, s = (torch.cos(a) * m).to(x.dtype)[:, None], (torch.sin(a) * m).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        y[..., i], y[..., i + half] = u * c - v * s, v * c + u * s
    return y


def softmax_rows(s):
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def attend(q, k, v, scale, softcap=0.0, r1=None, r2=None):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv]; softcap: bound of the scores; r1, r2 [H]: r1 ln(1 + r2 distance) is taken off."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    out = torch.empty((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = q[:, h] @ k[:, h // per].T * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        if r1 is not None:
            s = s - r1[h] * torch.log(1 + r2[h] * back.clamp(min=0).to(s.dtype))
        out[:, h] = softmax_rows(s.masked_fill(back < 0, -math.inf)) @ v[:, h // per]
    return out


def causal_conv(u, w, bias=None):
    """u [T, channels], w [channels, taps]: the last column is the current row's."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                y[t] = y[t] + w[:, j] * u[t - taps + 1 + j]
    return y if bias is None else y + bias


def temperature(positions, coef, every):
    return torch.tensor([1 + coef * math.log((int(p) + 1) // every + 1) for p in positions], dtype=torch.float64)


def project(x, w, p):
    return x @ w[p].T + w[p + ".b"]


def conv_attention(x, w, p, m, eps, kv=None):
    """(output, (keys, values)); `kv`: another layer's, used instead of own ones."""
    T, H, G = x.shape[0], m["heads"], m["kv_heads"]

    def part(c):
        y = project(x, w, p + c)
        return causal_conv(y, w[p + c + ".conv"]) if p + c + ".conv" in w else y
    q = unit_rms(part("q"), eps) * w[p + "q.norm"]
    if m.get("q_temp"):
        q = q * temperature(range(T), m["q_temp"]["coef"], m["q_temp"]["every"]).to(x.dtype)[:, None]
    if kv is None:
        k = unit_rms(part("k"), eps) * w[p + "k.norm"]
        kv = k.view(T, G, m["dim"]), part("v").view(T, G, m["vdim"])
    o = attend(q.view(T, H, m["dim"]), *kv, m["scale"], r1=w[p + "r1"], r2=w[p + "r2"])
    return project(o.reshape(T, -1), w, p + "o"), kv


def key_value_attention(x, w, p, m, eps):
    """Attention whose values are its keys in front of norm and rotation."""
    T, H, G, n = x.shape[0], m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(T)
    v = (x @ w[p + "k"].T).view(T, G, n)
    q = rotate(unit_rms((x @ w[p + "q"].T).view(T, H, n), eps) * w[p + "q.norm"], pos, m["rot"])
    k = rotate(unit_rms(v, eps) * w[p + "k.norm"], pos, m["rot"])
    return attend(q, k, v, m["scale"], m.get("softcap") or 0.0).reshape(T, -1) @ w[p + "o"].T


def scan(x, dt, B, C, A, D):
    """x, dt [T, c], B, C [T, n], A [c, n], D [c]: y [T, c]."""
    S = torch.zeros_like(A)
    y = torch.empty_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def selective_scan(h, w, p, m):
    inner, n, r = m["inner"], m["state"], m["dt_rank"]
    both = h @ w[p + "in"].T
    x = silu(causal_conv(both[:, :inner], w[p + "conv"], w[p + "conv.b"]))
    low = x @ w[p + "x"].T
    dt = softplus(low[:, :r] @ w[p + "dt"].T + w[p + "dt.b"])
    y = scan(x, dt, low[:, r:r + n], low[:, r + n:r + 2 * n], -torch.exp(w[p + "A_log"]), w[p + "D"])
    return (y * silu(both[:, inner:])) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    return m["left_scale"] * key_value_attention(h, w, p + "left.", m["left"], eps) + m["right_scale"] * selective_scan(h, w, p + "right.", m["right"])


def retain(q, k, v, decay):
    """q, k [T, H, n], v [T, H, dv]: S <- decay S + k v^T, o = S^T q."""
    T, H, _ = q.shape
    o = torch.empty_like(v)
    for h in range(H):
        S = torch.zeros((q.shape[2], v.shape[2]), dtype=v.dtype)
        for t in range(T):
            S = decay[h] * S + k[t, h][:, None] * v[t, h][None, :]
            o[t, h] = q[t, h] @ S
    return o


def retention(x, w, p, m, eps):
    T, H, n = x.shape[0], m["heads"], m["dim"]
    pos = torch.arange(T)
    q = rotate((x @ w[p + "q"].T).view(T, H, n), pos, m["rot"])
    k = rotate((x @ w[p + "k"].T).view(T, H, n), pos, m["rot"]) * n ** -0.5
    o = unit_rms(retain(q, k, (x @ w[p + "v"].T).view(T, H, m["vdim"]), m["decay"]), eps)
    return (o.reshape(T, -1) * silu(x @ w[p + "g"].T)) @ w[p + "o"].T


def relu2_ff(x, w, p):
    return torch.relu(x @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def expert(x, w, p):
    return (silu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def choose(z, top):
    """One token's experts: (indices, weights) from router logits z [E]."""
    s = sigmoid(z)
    idx = sorted(range(z.numel()), key=lambda e: -float(s[e]))[:top]
    return idx, s[idx]


def routed_ff(x, w, p, f):
    z = x @ w[p + "router"].T
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        idx, ws = choose(z[t], f["router"]["top"])
        for e, we in zip(idx, ws):
            out[t] += expert(we * x[t], w, f"{p}e{e}.")
    return out


def scalar_norm(x, g, eps):
    return unit_rms(x, eps) * g.reshape(())


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; `layers_out` (a list) receives the residual after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    kept = {}
    for i, e in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", e["mixer"], e.get("mlp")
        h = scalar_norm(x, w[p + "norm1"], eps)
        if e["type"] == "attention":
            y, kept[i] = conv_attention(h, w, p + "mix.", m, eps, kept[m["kv_from"]] if m.get("kv_from") is not None else None)
        elif e["type"] == "parallel":
            y = parallel(h, w, p + "mix.", m, eps)
        else:
            y = retention(h, w, p + "mix.", m, eps)
        x = x + y
        if f is not None:
            h = scalar_norm(x, w[p + "norm2"], eps)
            x = x + (relu2_ff(h, w, p + "mlp.") if f["kind"] == "dense" else routed_ff(h, w, p + "mlp.", f))
        if layers_out is not None:
            layers_out.append(x)
    return scalar_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
