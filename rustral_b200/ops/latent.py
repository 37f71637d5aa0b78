"""Latent attention ops: keys and values of all heads come from one cached vector per token, beside a rotated key part that the heads
share.  A slot of the cache holds [vector (rank) | rotated part]."""
from __future__ import annotations

import torch

from .. import _native as N
from .norm import norm_forward
from .paged import paged_attention_rows
from .rotary import rotate_pairs

N.optional_sig("rb_latent_prep", [N.C.POINTER(N.RbLatentPrepArgs), N.c_void_p])
N.optional_sig("rb_head_product", [N.C.POINTER(N.RbHeadProductArgs), N.c_void_p])
N.optional_sig("rb_latent_decode", [N.C.POINTER(N.RbLatentDecodeArgs), N.c_void_p])
N.optional_sig("rb_latent_decode_scratch_floats", [N.c_int, N.c_int, N.c_int, N.c_int, N.c_int], N.c_ll)
N._LAUNCHES["rb_latent_decode"] = 2


def latent_prep_(p, off_q: int, q_rank: int, off_kv: int, rank: int, rot: int, *, q_gamma, kv_gamma, eps: float, table, cache=None,
                 slots=None):
    """In place on the packed projection p [tokens, ..]: RMS norms (fp32 weights) of the query latent (columns off_q ..) and of the
    cached vector (off_kv ..), rotary positions (`table`, see rotary_table) on the `rot` columns behind it; vector and rotated part are
    stored in their cache slots (`cache` [blocks, block_size, 1, rank + rot])."""
    T = p.shape[0]
    if not p.is_cuda:
        for lo, n, g in ((off_q, q_rank, q_gamma), (off_kv, rank, kv_gamma)):
            p[:, lo:lo + n] = norm_forward(p[:, lo:lo + n].float(), g, None, eps, True)[0].to(p.dtype)
        kr = p[:, None, off_kv + rank:off_kv + rank + rot]
        p[:, off_kv + rank:off_kv + rank + rot] = rotate_pairs(kr, table)[:, 0]
        if cache is not None:
            keep = slots >= 0
            cache.view(-1, rank + rot)[slots[keep]] = p[:, off_kv:off_kv + rank + rot][keep].to(cache.dtype)
        return p
    a = N.RbLatentPrepArgs()
    a.p, a.ld, a.f32, a.tokens = p.data_ptr(), p.stride(0), int(p.dtype == torch.float32), T
    a.q_gamma, a.kv_gamma, a.table, a.pairs = q_gamma.data_ptr(), kv_gamma.data_ptr(), table.data_ptr(), table.shape[1]
    a.off_q, a.q_rank, a.off_kv, a.rank, a.rot, a.eps = off_q, q_rank, off_kv, rank, rot, eps
    if cache is not None:
        a.cache, a.slots, a.num_slots = cache.data_ptr(), slots.data_ptr(), cache.shape[0] * cache.shape[1]
    N.check(N.kernels().rb_latent_prep(a, N.stream_ptr()), "rb_latent_prep")
    return p


def head_product(x, x_head: int, w, heads: int, n: int, k: int, *, transposed: bool, gate=None, tail: int = 0, table=None,
                 out=None):
    """One small product per head.  x [rows, heads * x_head]: y[t, h, j] = sum_i x[t, h, i] w[h](j, i) over the first k numbers of the
    head; `w` holds the heads' matrices one below the other, [heads * n, k], or [heads * k, n] with `transposed`.  `gate`
    [rows, heads * n]: y times sigmoid(gate).  `tail`: that many numbers behind the head's first k are put behind y's n, their first
    pairs rotated by `table`.  Returns [rows, heads * (n + tail)] (`out`, row-strided views allowed)."""
    rows = x.shape[0]
    y = out if out is not None else torch.empty((rows, heads * (n + tail)), dtype=x.dtype, device=x.device)
    if rows == 0:
        return y
    if not x.is_cuda:
        x3 = x.reshape(rows, heads, x_head)
        w3 = w.float().reshape(heads, k, n) if transposed else w.float().reshape(heads, n, k).transpose(1, 2)
        y3 = torch.einsum("thk,hkn->thn", x3[..., :k].float(), w3)
        if gate is not None:
            y3 = y3 * torch.sigmoid(gate.float().reshape(rows, heads, n))
        y3 = y3.to(x.dtype)
        if tail:
            y3 = torch.cat([y3, rotate_pairs(x3[..., k:k + tail], table)], -1)
        return y.copy_(y3.reshape(rows, -1))
    a = N.RbHeadProductArgs()
    a.x, a.ld_x, a.x_head = x.data_ptr(), x.stride(0), x_head
    a.w, a.ld_w, a.w_head = w.data_ptr(), w.stride(0), w.stride(0) * (k if transposed else n)
    a.y, a.ld_y, a.y_head = y.data_ptr(), y.stride(0), n + tail
    if gate is not None:
        a.gate, a.ld_g = gate.data_ptr(), gate.stride(0)
    a.f32, a.rows, a.heads, a.n, a.k, a.transposed = int(x.dtype == torch.float32), rows, heads, n, k, int(transposed)
    if tail:
        a.tail, a.tail_off = tail, k
        if table is not None and table.shape[1]:
            a.table, a.pairs = table.data_ptr(), table.shape[1]
    N.check(N.kernels().rb_head_product(a, N.stream_ptr()), "rb_head_product")
    return y


def latent_decode_supported(q, rank: int, rot: int) -> bool:
    if not q.is_cuda:
        return True
    return q.dtype == torch.bfloat16 and rank % 8 == 0 and rot % 8 == 0 and rank <= 512 and rank + rot <= 640


def latent_decode(q, cache, rank: int, block_tables, context_lens, scale: float):
    """One token per sequence.  q [batch, heads * (rank + rot)]; cache [blocks, block_size, 1, rank + rot].  Returns the softmax-weighted
    sums of the cached vectors, [batch, heads * rank]."""
    nb, bs, _, width = cache.shape
    B, heads = q.shape[0], q.shape[1] // width
    if not q.is_cuda:
        return paged_attention_rows(q, cache, cache[..., :rank], block_tables, torch.arange(B), context_lens.long() - 1, scale)
    lib = N.kernels()
    out = torch.empty((B, heads * rank), dtype=q.dtype, device=q.device)
    scratch = torch.empty(lib.rb_latent_decode_scratch_floats(B, heads, rank, block_tables.shape[1], bs), dtype=torch.float32,
                          device=q.device)
    a = N.RbLatentDecodeArgs()
    a.q, a.ld_q, a.out, a.ld_o, a.cache, a.scratch = q.data_ptr(), q.stride(0), out.data_ptr(), out.stride(0), cache.data_ptr(), scratch.data_ptr()
    a.block_tables, a.max_blocks, a.context_lens = block_tables.data_ptr(), block_tables.shape[1], context_lens.data_ptr()
    a.num_blocks, a.block_size, a.batch, a.heads, a.rank, a.rot, a.scale = nb, bs, B, heads, rank, width - rank, scale
    N.check(lib.rb_latent_decode(a, N.stream_ptr()), "rb_latent_decode")
    return out
