"""Paged KV-cache ops: append and decode attention through a block table."""
from __future__ import annotations

import math

import torch

from .. import _native as N
from .attention import ScoreRule, attention_reference

N.optional_sig("rb_kv_append", [N.c_void_p, N.c_ll, N.c_void_p, N.c_ll, N.c_void_p, N.c_void_p, N.c_void_p, N.c_ll, N.c_int,
                                N.c_int, N.c_ll, N.c_void_p])
N.optional_sig("rb_paged_attention_decode", [N.c_void_p, N.c_ll, N.c_void_p, N.c_ll, N.c_void_p, N.c_void_p, N.c_void_p,
                                             N.c_int, N.c_void_p, N.c_int, N.c_int, N.c_int, N.c_int, N.c_int, N.c_ll,
                                             N.c_float, N.c_void_p, N.c_void_p])
N.optional_sig("rb_paged_attention_decode_rule", [N.C.POINTER(N.RbPagedDecodeArgs), N.c_void_p])
N._LAUNCHES["rb_paged_attention_decode_rule"] = 2
N.optional_sig("rb_paged_attention_scratch_floats", [N.c_int, N.c_int, N.c_int, N.c_int, N.c_int], N.c_ll)
N._LAUNCHES["rb_paged_attention_decode"] = 2


def kv_append(k_new, v_new, k_cache, v_cache, slot_mapping):
    """k_new / v_new: [tokens, kv_heads * head_dim] (row-strided views allowed); caches: [blocks, block_size, kv_heads, D];
    slot_mapping: int64 [tokens] = block * block_size + offset (negative = skip)."""
    tokens = k_new.shape[0]
    nb, bs, hk, d = k_cache.shape
    if not k_new.is_cuda:
        kc, vc = k_cache.view(nb * bs, hk * d), v_cache.view(nb * bs, hk * d)
        ok = slot_mapping >= 0
        kc[slot_mapping[ok]] = k_new[ok].to(kc.dtype)
        vc[slot_mapping[ok]] = v_new[ok].to(vc.dtype)
        return
    N.check(N.kernels().rb_kv_append(k_new.data_ptr(), k_new.stride(0), v_new.data_ptr(), v_new.stride(0), k_cache.data_ptr(),
                                     v_cache.data_ptr(), slot_mapping.data_ptr(), tokens, hk, d, nb * bs, N.stream_ptr()),
            "rb_kv_append")


def decode_supported(q, dk: int, dv: int, rule: ScoreRule | None = None, gate=None) -> bool:
    """Whether `paged_attention_decode` takes these operands."""
    if not q.is_cuda:
        return True
    if q.dtype != torch.bfloat16:
        return False
    if rule is None and gate is None and dk == dv:
        return dk in (64, 128)
    return dk % 8 == 0 and dv % 8 == 0 and max(dk, dv) <= 128 and q.stride(0) % 2 == 0 and q.data_ptr() % 4 == 0


def paged_attention_decode(q, k_cache, v_cache, block_tables, context_lens, scale=None, out=None, rule: ScoreRule | None = None,
                           gate=None, head_gate=None):
    """q: [batch, heads * dk] (or [batch, heads, dk]); block_tables int32 [batch, max_blocks]; context_lens int32 [batch].
    Returns [batch, heads * dv].  `rule`: see ops.ScoreRule; `gate` [batch, heads * dv] or `head_gate` fp32 [batch, heads]: the
    output times sigmoid(gate)."""
    nb, bs, hk, d = k_cache.shape
    dv = v_cache.shape[3]
    B = q.shape[0]
    q2 = q.reshape(B, -1)
    heads = q2.shape[1] // d
    scale = 1.0 / math.sqrt(d) if scale is None else scale
    plain = rule is None and gate is None and head_gate is None and dv == d
    if not q.is_cuda and not plain:
        return paged_attention_rows(q2, k_cache, v_cache, block_tables, torch.arange(B), context_lens.long() - 1, scale, rule, gate, out,
                                    head_gate)
    if not q.is_cuda:
        o = torch.zeros(B, heads, d)
        kc, vc = k_cache.view(nb * bs, hk, d).float(), v_cache.view(nb * bs, hk, d).float()
        for b in range(B):
            n = int(context_lens[b])
            toks = torch.arange(n)
            slots = block_tables[b, toks // bs].long() * bs + toks % bs
            kk = kc[slots].repeat_interleave(heads // hk, 1)          # [n, heads, d]
            vv = vc[slots].repeat_interleave(heads // hk, 1)
            s = torch.einsum("hd,nhd->hn", q2[b].float().view(heads, d), kk) * scale
            o[b] = torch.einsum("hn,nhd->hd", torch.softmax(s, -1), vv)
        r = o.reshape(B, heads * d).to(q.dtype)
        if out is not None:
            out.copy_(r)
            return out
        return r
    out = out if out is not None else torch.empty((B, heads * dv), dtype=q.dtype, device=q.device)
    lib = N.kernels()
    scratch = torch.empty(lib.rb_paged_attention_scratch_floats(B, heads, dv, block_tables.shape[1], bs), dtype=torch.float32,
                          device=q.device)
    if not plain:
        rule = rule or ScoreRule()
        a = N.RbPagedDecodeArgs()
        a.q, a.ld_q, a.out, a.ld_o = q2.data_ptr(), q2.stride(0), out.data_ptr(), out.stride(0)
        a.k_cache, a.v_cache, a.num_blocks, a.block_size = k_cache.data_ptr(), v_cache.data_ptr(), nb, bs
        a.block_tables, a.max_blocks, a.context_lens = block_tables.data_ptr(), block_tables.shape[1], context_lens.data_ptr()
        if gate is not None:
            a.gate, a.ld_g = gate.data_ptr(), gate.stride(0)
        if head_gate is not None:
            a.head_gate, a.ld_g = head_gate.data_ptr(), head_gate.stride(0)
        a.window, a.keep_first, a.sink = rule.window, rule.keep_first, int(rule.sink)
        a.log_amount, a.log_rate, a.out_scale = N.ptr(rule.log_amount), N.ptr(rule.log_rate), rule.out_scale
        a.scratch, a.batch, a.heads, a.kv_heads, a.dk, a.dv = scratch.data_ptr(), B, heads, hk, d, dv
        a.scale, a.softcap, a.slopes, a.chunk = scale, rule.softcap, N.ptr(rule.slopes), rule.chunk
        N.check(lib.rb_paged_attention_decode_rule(a, N.stream_ptr()), "rb_paged_attention_decode_rule")
        return out
    N.check(lib.rb_paged_attention_decode(q2.data_ptr(), q2.stride(0), out.data_ptr(), out.stride(0),
                                          k_cache.data_ptr(), v_cache.data_ptr(), block_tables.data_ptr(),
                                          block_tables.shape[1], context_lens.data_ptr(), B, heads, hk, d, bs, nb,
                                          scale, scratch.data_ptr(), N.stream_ptr()), "rb_paged_attention_decode")
    return out


N.optional_sig("rb_paged_attention_rows", [N.C.POINTER(N.RbPagedRowsArgs), N.c_void_p])


def paged_attention_rows(q, k_cache, v_cache, block_tables, row_seq, row_pos, scale: float, rule: ScoreRule | None = None,
                         gate=None, out=None, head_gate=None):
    """Attention over the pages for any rows of a batch.  q: [rows, heads * dk] (row-strided views allowed); row r is the
    token at position row_pos[r] (int64) of the sequence with pages block_tables[row_seq[r]] (int32); its own key is
    already in the cache.  Takes bf16 and fp32 and any head sizes; `v_cache` may be the first columns of `k_cache`.  `gate` [rows, heads * dv] or `head_gate` fp32 [rows, heads]:
    output times sigmoid(gate)."""
    nb, bs, hk, dk = k_cache.shape
    dv = v_cache.shape[3]
    rows, heads = q.shape[0], q.shape[1] // dk
    rule = rule or ScoreRule()
    out = out if out is not None else torch.empty((rows, heads * dv), dtype=q.dtype, device=q.device)
    if not q.is_cuda:
        kc, vc = k_cache.view(nb * bs, hk, dk), v_cache.reshape(nb * bs, hk, dv)
        for r in range(rows):
            n, table = int(row_pos[r]) + 1, block_tables[int(row_seq[r])].long()
            kept, lo = rule.key_ranges(n - 1)
            toks = torch.cat([torch.arange(kept), torch.arange(lo, n)])
            slots = table[toks // bs] * bs + toks % bs
            o = attention_reference(q[r].view(1, 1, heads, dk), kc[slots][None], vc[slots][None], True, scale, rule=rule)
            o = o.reshape(-1).float()
            if head_gate is not None:
                o = (o.view(heads, dv) * torch.sigmoid(head_gate[r].float())[:, None]).reshape(-1)
            out[r] = o * torch.sigmoid(gate[r].float()) if gate is not None else o
        return out
    a = N.RbPagedRowsArgs()
    a.q, a.ld_q, a.out, a.ld_o = q.data_ptr(), q.stride(0), out.data_ptr(), out.stride(0)
    a.k_cache, a.v_cache, a.num_blocks, a.block_size = k_cache.data_ptr(), v_cache.data_ptr(), nb, bs
    a.ld_kc, a.ld_vc = k_cache.stride(1), v_cache.stride(1)
    a.block_tables, a.max_blocks = block_tables.data_ptr(), block_tables.shape[1]
    a.row_seq, a.row_pos = row_seq.data_ptr(), row_pos.data_ptr()
    if gate is not None:
        a.gate, a.ld_g = gate.data_ptr(), gate.stride(0)
    if head_gate is not None:
        a.head_gate, a.ld_g = head_gate.data_ptr(), head_gate.stride(0)
    a.window, a.keep_first, a.sink = rule.window, rule.keep_first, int(rule.sink)
    a.log_amount, a.log_rate, a.out_scale = N.ptr(rule.log_amount), N.ptr(rule.log_rate), rule.out_scale
    a.f32, a.rows, a.heads, a.kv_heads, a.dk, a.dv = int(q.dtype == torch.float32), rows, heads, hk, dk, dv
    a.scale, a.softcap, a.slopes, a.chunk = scale, rule.softcap, N.ptr(rule.slopes), rule.chunk
    N.check(N.kernels().rb_paged_attention_rows(a, N.stream_ptr()), "rb_paged_attention_rows")
    return out
