"""Work between a packed attention projection and the attention kernels: query / key norm (per head or over the whole projection), rotary
positions, query temperature, value mixing, cache append."""
from __future__ import annotations

import torch

from .. import _native as N
from .rotary import rotate_halves, rotate_pairs

N.optional_sig("rb_head_prep", [N.C.POINTER(N.RbHeadPrepArgs), N.c_void_p])


def head_prep_(p, heads: int, kv_heads: int, dk: int, dv: int, *, q_gamma=None, k_gamma=None, eps: float = 1e-5, v_first=None,
               mix=None, k_cache=None, v_cache=None, slots=None, rot=None, half: bool = False, k_scale: float = 1.0,
               q_col: int = 0, k_col: int | None = None, v_col: int | None = None, values_are_keys: bool = False):
    """In place on `p` = [q | k | v | ...] ([tokens, >= heads * dk + kv_heads * (dk + dv)]): every query and key head gets an
    RMS norm (weights `q_gamma` / `k_gamma` [dk], None: no norm) and rotary positions (`rot`: fp32 [tokens, pairs, 2] of
    `rotary_table`, on the first 2 * pairs numbers), the values become (1 - mix) v + mix v_first (`v_first`:
    [tokens, kv_heads * dv], `mix` fp32 [1]; None: unchanged), and keys and values are stored in their cache slots.

    `half`: numbers i and i + pairs turn together instead of neighbours; keys are then multiplied by `k_scale`, and with
    `values_are_keys` the value columns receive the keys as they were.  `q_col`, `k_col`, `v_col`: first columns of the parts."""
    T = p.shape[0]
    ok = heads * dk if k_col is None else k_col
    ov = (heads + kv_heads) * dk if v_col is None else v_col
    end = ov + kv_heads * dv
    if not half and (k_scale != 1.0 or values_are_keys):
        raise ValueError("head_prep: k_scale and values_are_keys come with halves that turn")
    if half and (v_first is not None or (values_are_keys and dk != dv)):
        raise ValueError("head_prep: no value mixing with halves that turn, and values that are keys have their size")
    if not p.is_cuda:
        if values_are_keys:
            p[:, ov:end] = p[:, ok:ok + kv_heads * dk]
        for lo, n, g in ((q_col, heads, q_gamma), (ok, kv_heads, k_gamma)):
            if g is not None:
                x = p[:, lo:lo + n * dk].float().view(T, n, dk)
                x = x * torch.rsqrt((x * x).mean(-1, keepdim=True) + eps) * g.float()
                p[:, lo:lo + n * dk] = x.reshape(T, n * dk).to(p.dtype)
            if rot is not None:
                x = p[:, lo:lo + n * dk].reshape(T, n, dk)
                p[:, lo:lo + n * dk] = (rotate_halves if half else rotate_pairs)(x, rot).reshape(T, n * dk)
        if k_scale != 1.0:
            p[:, ok:ok + kv_heads * dk] = (p[:, ok:ok + kv_heads * dk].float() * k_scale).to(p.dtype)
        if v_first is not None:
            lam = mix.float()
            p[:, ov:end] = ((1 - lam) * p[:, ov:end].float() + lam * v_first.float()).to(p.dtype)
        if k_cache is not None:
            nb, bs = k_cache.shape[:2]
            keep = slots >= 0
            k_cache.view(nb * bs, kv_heads * dk)[slots[keep]] = p[:, ok:ok + kv_heads * dk][keep].to(k_cache.dtype)
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
    a.off_q, a.off_k, a.off_v, a.tokens = q_col, ok, ov, T
    a.half, a.k_scale, a.values_are_keys = int(half), k_scale, int(values_are_keys)
    a.heads, a.kv_heads, a.dk, a.dv, a.eps = heads, kv_heads, dk, dv, eps
    N.check(N.kernels().rb_head_prep(a, N.stream_ptr()), "rb_head_prep")
    return p


N.optional_sig("rb_row_prep", [N.C.POINTER(N.RbRowPrepArgs), N.c_void_p])


def row_prep_(p, heads: int, kv_heads: int, dk: int, dv: int, *, q_gamma, k_gamma=None, eps: float = 1e-5, pos=None, temp_coef: float = 0.0,
              temp_every: int = 0, k_cache=None, v_cache=None, slots=None):
    """In place on `p` = [q | k | v] ([tokens, heads * dk + kv_heads * (dk + dv)], or with kv_heads 0 the queries alone): all queries of
    a token get one RMS norm over the whole row (weight `q_gamma` fp32 [heads * dk]) and so do its keys (`k_gamma`); with `temp_every`
    the queries are multiplied by 1 + temp_coef * ln(floor((pos + 1) / temp_every) + 1) (`pos` int64 [tokens]); keys and values are stored
    in their cache slots."""
    T = p.shape[0]
    ok, ov = heads * dk, (heads + kv_heads) * dk
    end = ov + kv_heads * dv
    if not p.is_cuda:
        for lo, hi, g in ((0, ok, q_gamma), (ok, ov, k_gamma)):
            if hi > lo:
                x = p[:, lo:hi].float()
                x = x * torch.rsqrt((x * x).mean(-1, keepdim=True) + eps) * g.float()
                if lo == 0 and temp_every:
                    x = x * (1.0 + temp_coef * torch.log(((pos + 1) // temp_every + 1).float()))[:, None]
                p[:, lo:hi] = x.to(p.dtype)
        if k_cache is not None and kv_heads:
            keep = slots >= 0
            k_cache.view(-1, kv_heads * dk)[slots[keep]] = p[:, ok:ov][keep].to(k_cache.dtype)
            v_cache.view(-1, kv_heads * dv)[slots[keep]] = p[:, ov:end][keep].to(v_cache.dtype)
        return p
    a = N.RbRowPrepArgs()
    a.p, a.ld, a.f32, a.tokens, a.eps = p.data_ptr(), p.stride(0), int(p.dtype == torch.float32), T, eps
    a.nq, a.nk, a.nv = ok, kv_heads * dk, kv_heads * dv
    a.q_gamma, a.k_gamma = q_gamma.data_ptr(), N.ptr(k_gamma)
    if temp_every:
        a.pos, a.temp_coef, a.temp_every = pos.data_ptr(), temp_coef, temp_every
    if k_cache is not None and kv_heads:
        a.k_cache, a.v_cache, a.slots = k_cache.data_ptr(), v_cache.data_ptr(), slots.data_ptr()
        a.num_slots = k_cache.shape[0] * k_cache.shape[1]
    N.check(N.kernels().rb_row_prep(a, N.stream_ptr()), "rb_row_prep")
    return p
