"""Per-head work between a packed attention projection and the attention kernels: query / key norm, rotary positions, value mixing,
cache append."""
from __future__ import annotations

import torch

from .. import _native as N
from .rotary import rotate_pairs

N.optional_sig("rb_head_prep", [N.C.POINTER(N.RbHeadPrepArgs), N.c_void_p])


def head_prep_(p, heads: int, kv_heads: int, dk: int, dv: int, *, q_gamma=None, k_gamma=None, eps: float = 1e-5, v_first=None,
               mix=None, k_cache=None, v_cache=None, slots=None, rot=None):
    """In place on `p` = [q | k | v | ...] ([tokens, >= heads * dk + kv_heads * (dk + dv)]): every query and key head gets an
    RMS norm (weights `q_gamma` / `k_gamma` [dk], None: no norm) and rotary positions (`rot`: fp32 [tokens, pairs, 2] of
    `rotary_table`, on the first 2 * pairs numbers), the values become (1 - mix) v + mix v_first (`v_first`:
    [tokens, kv_heads * dv], `mix` fp32 [1]; None: unchanged), and keys and values are stored in their cache slots."""
    T = p.shape[0]
    ok, ov = heads * dk, (heads + kv_heads) * dk
    end = ov + kv_heads * dv
    if not p.is_cuda:
        for lo, n, g in ((0, heads, q_gamma), (ok, kv_heads, k_gamma)):
            if g is not None:
                x = p[:, lo:lo + n * dk].float().view(T, n, dk)
                x = x * torch.rsqrt((x * x).mean(-1, keepdim=True) + eps) * g.float()
                p[:, lo:lo + n * dk] = x.reshape(T, n * dk).to(p.dtype)
            if rot is not None:
                x = p[:, lo:lo + n * dk].reshape(T, n, dk)
                p[:, lo:lo + n * dk] = rotate_pairs(x, rot).reshape(T, n * dk)
        if v_first is not None:
            lam = mix.float()
            p[:, ov:end] = ((1 - lam) * p[:, ov:end].float() + lam * v_first.float()).to(p.dtype)
        if k_cache is not None:
            nb, bs = k_cache.shape[:2]
            keep = slots >= 0
            k_cache.view(nb * bs, kv_heads * dk)[slots[keep]] = p[:, ok:ov][keep].to(k_cache.dtype)
            v_cache.view(nb * bs, kv_heads * dv)[slots[keep]] = p[:, ov:end][keep].to(v_cache.dtype)
        return p
    a = N.RbHeadPrepArgs()
    a.p, a.ld, a.f32 = p.data_ptr(), p.stride(0), int(p.dtype == torch.float32)
    a.q_gamma, a.k_gamma = N.ptr(q_gamma), N.ptr(k_gamma)
    if v_first is not None:
        a.v_first, a.ld_vf, a.mix = v_first.data_ptr(), v_first.stride(0), mix.data_ptr()
    if k_cache is not None:
        a.k_cache, a.v_cache, a.slots = k_cache.data_ptr(), v_cache.data_ptr(), slots.data_ptr()
        a.num_slots = k_cache.shape[0] * k_cache.shape[1]
    if rot is not None:
        a.rot, a.rot_dims = rot.data_ptr(), 2 * rot.shape[1]
    a.off_q, a.off_k, a.off_v, a.tokens = 0, ok, ov, T
    a.heads, a.kv_heads, a.dk, a.dv, a.eps = heads, kv_heads, dk, dv, eps
    N.check(N.kernels().rb_head_prep(a, N.stream_ptr()), "rb_head_prep")
    return p
