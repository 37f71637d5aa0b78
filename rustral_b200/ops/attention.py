"""Flash attention (causal / full, MHA / GQA) with a differentiable wrapper and a plain reference."""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from .. import _native as N


@dataclass(frozen=True, eq=False)
class ScoreRule:
    """What happens to scaled attention scores before the softmax, and which keys a query sees besides causality.

    softcap > 0: score <- softcap * tanh(score / softcap).  slopes (fp32 [heads]): score <- score - slopes[h] * (i - j), after
    the cap.  chunk > 0: position i sees j only when i // chunk == j // chunk (positions of the sequence; a kernel that is
    handed keys from a chunk's first one on may count from there).  window > 0: position i sees j only when i - j < window or
    j < keep_first (a kernel may be handed the kept keys and then those from the first query's window on).  sink: a further
    score 0 without a value takes part in the softmax.  log_amount, log_rate (fp32 [heads] each): score <- score - log_amount[h] *
    ln(1 + log_rate[h] * (i - j)), after the cap.  out_scale multiplies the output."""
    softcap: float = 0.0
    slopes: torch.Tensor | None = None
    chunk: int = 0
    window: int = 0
    keep_first: int = 0
    sink: bool = False
    log_amount: torch.Tensor | None = None
    log_rate: torch.Tensor | None = None
    out_scale: float = 1.0

    def first_key(self, pos: int) -> int:
        """The first position that the token at `pos` can see, apart from the kept ones."""
        if self.window:
            return max(0, pos - self.window + 1)
        return pos // self.chunk * self.chunk if self.chunk else 0

    def key_ranges(self, pos: int) -> tuple:
        """(kept, first): the token at `pos` and those behind it need the keys [0, kept) and [first, ...)."""
        first = self.first_key(pos)
        kept = self.keep_first if self.window else 0
        if kept and (self.slopes is not None or self.log_rate is not None):
            first = 0                                         # a distance bias wants the keys without a gap
        return (0, 0) if first <= kept else (kept, first)

    @property
    def plain(self) -> bool:
        return not self.softcap and self.slopes is None and not self.chunk and not self.window and not self.sink and \
            self.log_rate is None and self.out_scale == 1.0


def softmax_with_sink(s: torch.Tensor) -> torch.Tensor:
    """Softmax over the last dimension with a further score 0 whose weight is dropped."""
    return torch.softmax(torch.cat([s, torch.zeros_like(s[..., :1])], -1), -1)[..., :-1]


def distance_slopes(heads: int, device=None) -> torch.Tensor:
    """Per-head slopes of a linear distance bias: the geometric sequence 2^(-8 (h + 1) / heads)."""
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float32, device=device)


def attention_reference(q, k, v, causal: bool, scale: float | None = None, kv_lens=None, rule: ScoreRule | None = None):
    """fp32 softmax(QK^T * scale + mask) V on [B, S, H, D] tensors (GQA: fewer K/V heads; V may have its own head size).
    `kv_lens` ([B] integers): keys at positions >= kv_lens[b] are padding (a batch entry without any real key gives zero
    rows).  `rule`: see ScoreRule; key 0 is taken as the start of a chunk."""
    B, Sq, H, D = q.shape
    Sk, Hk = k.shape[1], k.shape[2]
    scale = 1.0 / math.sqrt(D) if scale is None else scale
    qf = q.float().permute(0, 2, 1, 3)
    kf, vf = k.float().permute(0, 2, 1, 3), v.float().permute(0, 2, 1, 3)
    if H != Hk:                                             # grouped-query attention: every K/V head serves H / Hk query heads
        kf, vf = kf.repeat_interleave(H // Hk, dim=1), vf.repeat_interleave(H // Hk, dim=1)
    s = qf @ kf.transpose(-1, -2) * scale
    i = torch.arange(Sq, device=q.device)[:, None] + (Sk - Sq)
    j = torch.arange(Sk, device=q.device)[None, :]
    if rule is not None:
        if rule.softcap:
            s = rule.softcap * torch.tanh(s / rule.softcap)
        if rule.slopes is not None:
            s = s - rule.slopes.to(q.device).float()[None, :, None, None] * (i - j).float()
        if rule.log_rate is not None:
            r1, r2 = (t.to(q.device).float()[None, :, None, None] for t in (rule.log_amount, rule.log_rate))
            s = s - r1 * torch.log1p(r2 * (i - j).clamp(min=0).float())
        if rule.chunk:
            s = s.masked_fill(i // rule.chunk != j // rule.chunk, float("-inf"))
        if rule.window:
            s = s.masked_fill((i - j >= rule.window) & (j >= rule.keep_first), float("-inf"))
    if causal:
        s = s.masked_fill(j > i, float("-inf"))
    if kv_lens is not None:
        pad = torch.arange(Sk, device=q.device)[None, :] >= kv_lens.to(q.device).long()[:, None]      # [B, Sk]
        s = s.masked_fill(pad[:, None, None, :], float("-inf"))
    p = softmax_with_sink(s) if rule is not None and rule.sink else torch.softmax(s, -1)
    if kv_lens is not None:
        p = torch.nan_to_num(p, nan=0.0)                      # rows without a visible key
    o = (p @ vf).permute(0, 2, 1, 3)
    return (o if rule is None or rule.out_scale == 1.0 else o * rule.out_scale).to(q.dtype)


def _strides3(t):
    # [B, S, H, D] view -> element strides (batch, row, head)
    return (t.stride(0), t.stride(1), t.stride(2))


def _fill(args, q, k, v, o, causal, scale, kv_lens=None):
    B, Sq, H, D = q.shape
    if kv_lens is not None:
        if kv_lens.dtype != torch.int32 or not kv_lens.is_cuda or kv_lens.numel() != B or not kv_lens.is_contiguous():
            raise TypeError("attention: kv_lens must be a contiguous int32 CUDA tensor with one entry per batch element")
        args.kv_lens = kv_lens.data_ptr()
    else:
        args.kv_lens = None
    args.q, args.k, args.v, args.o = q.data_ptr(), k.data_ptr(), v.data_ptr(), o.data_ptr()
    for name, t in (("q_strides", q), ("k_strides", k), ("v_strides", v), ("o_strides", o)):
        st = _strides3(t)
        arr = getattr(args, name)
        arr[0], arr[1], arr[2] = st
    args.batch, args.heads, args.kv_heads = B, H, k.shape[2]
    args.seq_q, args.seq_k, args.head_dim = Sq, k.shape[1], D
    args.causal, args.scale = int(causal), scale


N.optional_sig("rb_attention_fwd_tc", [N.C.POINTER(N.RbAttnArgs), N.c_void_p])
N.optional_sig("rb_attention_bwd_tc", [N.C.POINTER(N.RbAttnArgs), N.c_void_p])
N.optional_sig("rb_attention_fwd_tc2", [N.C.POINTER(N.RbAttnArgs), N.c_int, N.c_void_p])
N.optional_sig("rb_attention_bwd_tc2", [N.C.POINTER(N.RbAttnArgs), N.c_void_p])
N._LAUNCHES["rb_attention_bwd_tc2"] = 3
N._LAUNCHES["rb_attention_bwd_tc"] = 3

# "tc2": tcgen05 kernel with two query tiles per CTA in ping-pong (falls back to "tc" for shapes it does not take);
# "tc": one query tile per CTA; "mma": the mma.sync kernel.
FORWARD_IMPL = __import__("os").environ.get("RUSTRAL_ATTN_IMPL", "tc2")
# Share of the exponentials the "tc2" kernel computes with a polynomial on the FMA pipe: 0 (none) or 4 (every fourth
# pair).  Measured on B200, batch 32 x 12 heads x 1024 x 64 / batch 4 x 32 (8 KV) heads x 4096 x 128: 0 -> 191 us / 732 us,
# 4 -> 218 / 847; the one-tile "tc" kernel 220 / 1492.
FORWARD_POLY_EVERY = int(__import__("os").environ.get("RUSTRAL_ATTN_POLY", "0"))
# Backward: "tc2" keeps P and dS in TMEM and feeds the dV / dK / dQ products from there; "tc" stages them through shared
# memory.  Measured on the same two shapes: tc2 497 us / 2502 us, tc 574 / 3146.
BACKWARD_IMPL = __import__("os").environ.get("RUSTRAL_ATTN_BWD_IMPL", "mma" if FORWARD_IMPL == "mma" else "tc2")


def attention_forward(q, k, v, causal: bool, scale: float, out=None, want_lse: bool = True, impl: str | None = None,
                      kv_lens=None):
    """q: [B, Sq, H, D]; k, v: [B, Sk, Hkv, D] (any strides with a contiguous D).  Returns (o, lse).  `kv_lens`
    (int32 [B] on the device): number of real keys per batch entry, the rest is padding (second-generation kernels)."""
    B, Sq, H, D = q.shape
    for t in (q, k, v):
        if t.dtype != torch.bfloat16 or t.stride(3) != 1:
            raise TypeError("attention: bf16 tensors with a contiguous head dimension are required")
    o = out if out is not None else torch.empty((B, Sq, H, D), dtype=q.dtype, device=q.device)
    lse = torch.empty((B, H, Sq), dtype=torch.float32, device=q.device) if want_lse else None
    a = N.RbAttnArgs()
    _fill(a, q, k, v, o, causal, scale, kv_lens)
    a.lse = N.ptr(lse)
    lib = N.kernels()
    which = impl or FORWARD_IMPL
    if kv_lens is not None and not which.startswith("tc2"):
        which = "tc2"
    if which.startswith("tc2") and hasattr(lib, "rb_attention_fwd_tc2"):
        poly = int(which[4:]) if len(which) > 4 else FORWARD_POLY_EVERY          # "tc2:4" selects the share explicitly
        rc = lib.rb_attention_fwd_tc2(a, poly, N.stream_ptr())
        if rc != -9:
            N.check(rc, "rb_attention_fwd_tc2")
            return o, lse
        which = "tc"
    if which == "tc" and hasattr(lib, "rb_attention_fwd_tc"):
        rc = lib.rb_attention_fwd_tc(a, N.stream_ptr())
        if rc != -9:
            N.check(rc, "rb_attention_fwd_tc")
            return o, lse
    N.check(lib.rb_attention_fwd(a, N.stream_ptr()), "rb_attention_fwd")
    return o, lse


def prompt_supported(q, k, v, dk: int, dv: int, rule: ScoreRule | None = None, gate=None) -> bool:
    """Whether `prompt_attention` takes these operands (2-D [rows, heads * size] views)."""
    if not q.is_cuda:
        return True
    if q.dtype != torch.bfloat16:
        return False
    if rule is None and gate is None and dk == dv:
        return dk in (64, 128)
    views = [t for t in (q, k, v, gate) if t is not None]
    return dk % 8 == 0 and dv % 8 == 0 and max(dk, dv) <= 128 and \
        all(t.stride(0) % 8 == 0 and t.data_ptr() % 16 == 0 for t in views)


N.optional_sig("rb_attention_fwd_rule", [N.C.POINTER(N.RbAttnArgs), N.C.POINTER(N.RbAttnRule), N.c_void_p])


def prompt_attention(q, k, v, scale: float, out, rule: ScoreRule | None = None, gate=None, head_gate=None):
    """Causal attention of a prompt portion in inference: q [1, L, H, dk], k [1, S, G, dk], v [1, S, G, dv] with the last L
    keys being the portion itself, out [1, L, H, dv].  `rule`: see ScoreRule (key 0 starts a chunk; with a window the keys may
    be those of `key_ranges`); `gate` [L, H * dv] or `head_gate` fp32 [L, H]: out <- out * sigmoid(gate)."""
    if not q.is_cuda:
        o = attention_reference(q, k, v, True, scale, rule=rule)
        if gate is not None:
            o = o.float() * torch.sigmoid(gate.float().reshape(o.shape))
        if head_gate is not None:
            o = o.float() * torch.sigmoid(head_gate.float())[None, :, :, None]
        out.copy_(o)
        return out
    dv = v.shape[3]
    if rule is None and gate is None and head_gate is None and dv == q.shape[3]:
        return attention_forward(q, k, v, True, scale, out=out, want_lse=False)[0]
    rule = rule or ScoreRule()
    a, r = N.RbAttnArgs(), N.RbAttnRule()
    _fill(a, q, k, v, out, True, scale)
    r.v_dim, r.softcap, r.slopes, r.chunk = dv, rule.softcap, N.ptr(rule.slopes), rule.chunk
    r.window, r.keep_first, r.sink = rule.window, rule.keep_first, int(rule.sink)
    r.log_amount, r.log_rate, r.out_scale = N.ptr(rule.log_amount), N.ptr(rule.log_rate), rule.out_scale
    if gate is not None:
        r.gate, r.ld_gate = gate.data_ptr(), gate.stride(0)
    if head_gate is not None:
        r.head_gate, r.ld_gate = head_gate.data_ptr(), head_gate.stride(0)
    N.check(N.kernels().rb_attention_fwd_rule(a, r, N.stream_ptr()), "rb_attention_fwd_rule")
    return out


def split_supported(dn: int, dr: int, dv: int, *views) -> bool:
    """Whether `prompt_attention_split` takes these head sizes and operands (2-D row-strided views; None: absent)."""
    views = [t for t in views if t is not None]
    if not views[0].is_cuda:
        return True
    if any(t.dtype != torch.bfloat16 or t.stride(0) % 8 or t.data_ptr() % 16 for t in views):
        return False
    return (dn | dr | dv) % 8 == 0 and max(dn, dv) <= 128 and dr <= 64


def prompt_attention_split(q, k, v, k_rot, scale: float, out, gate=None):
    """Causal attention of a prompt portion whose keys have a second part that all heads share: q [1, L, H, dn + dr], k [1, S, H, dn],
    k_rot [S, dr], v [1, S, H, dv], out [1, L, H, dv]; score = (q[:dn] . k + q[dn:] . k_rot) * scale.  `gate` [L, H * dv]: out <- out *
    sigmoid(gate).  On a GPU dr is at most 64 (bf16, sizes in multiples of 8, at most 128)."""
    dn, dv, dr = k.shape[3], v.shape[3], k_rot.shape[1]
    if not q.is_cuda:
        kk = torch.cat([k.float(), k_rot.float()[None, :, None, :].expand(1, k.shape[1], k.shape[2], dr)], -1)
        o = attention_reference(q.float(), kk, v, True, scale)
        out.copy_(o if gate is None else o * torch.sigmoid(gate.float().reshape(o.shape)))
        return out
    a, r = N.RbAttnArgs(), N.RbAttnRule()
    _fill(a, q[..., :dn], k, v, out, True, scale)
    r.out_scale = 1.0
    r.v_dim, r.rot_dim, r.k_rot, r.ld_k_rot = dv, dr, k_rot.data_ptr(), k_rot.stride(0)
    if gate is not None:
        r.gate, r.ld_gate = gate.data_ptr(), gate.stride(0)
    N.check(N.kernels().rb_attention_fwd_rule(a, r, N.stream_ptr()), "rb_attention_fwd_rule")
    return out


def attention_backward(do, q, k, v, o, lse, causal: bool, scale: float, dq=None, dk=None, dv=None, impl: str | None = None,
                       kv_lens=None):
    B, Sq, H, D = q.shape
    if do.stride(3) != 1 or _strides3(do) != _strides3(o):
        do = _match(do, o)
    dq = dq if dq is not None else torch.empty_like(q)
    dk = dk if dk is not None else torch.empty_like(k)
    dv = dv if dv is not None else torch.empty_like(v)
    delta = torch.empty((B, H, Sq), dtype=torch.float32, device=q.device)
    a = N.RbAttnArgs()
    _fill(a, q, k, v, o, causal, scale, kv_lens)
    a.d_o = do.data_ptr()
    a.dq, a.dk, a.dv = dq.data_ptr(), dk.data_ptr(), dv.data_ptr()
    for name, t in (("dq_strides", dq), ("dk_strides", dk), ("dv_strides", dv)):
        st = _strides3(t)
        arr = getattr(a, name)
        arr[0], arr[1], arr[2] = st
    a.lse, a.delta = lse.data_ptr(), delta.data_ptr()
    lib = N.kernels()
    which = "tc2" if kv_lens is not None else (impl or BACKWARD_IMPL)
    if which == "tc2" and hasattr(lib, "rb_attention_bwd_tc2"):     # P / dS kept in TMEM (falls back to "tc")
        rc = lib.rb_attention_bwd_tc2(a, N.stream_ptr())
        if rc != -9:
            N.check(rc, "rb_attention_bwd_tc2")
            return dq, dk, dv
        which = "tc"
    if which == "tc" and hasattr(lib, "rb_attention_bwd_tc"):
        rc = lib.rb_attention_bwd_tc(a, N.stream_ptr())
        if rc != -9:
            N.check(rc, "rb_attention_bwd_tc")
            return dq, dk, dv
    N.check(lib.rb_attention_bwd(a, N.stream_ptr()), "rb_attention_bwd")
    return dq, dk, dv


def _match(do, o):
    """A copy of `do` laid out with the strides of `o` (the kernel reads both with one stride set)."""
    buf = torch.empty_strided(o.shape, o.stride(), dtype=do.dtype, device=do.device)
    buf.copy_(do)
    return buf


class _FlashFn(torch.autograd.Function):
    @staticmethod
    def forward(ctx, q, k, v, causal, scale, kv_lens=None):
        o, lse = attention_forward(q, k, v, causal, scale, kv_lens=kv_lens)
        ctx.save_for_backward(q, k, v, o, lse)
        ctx.causal, ctx.scale, ctx.kv_lens = causal, scale, kv_lens
        return o

    @staticmethod
    def backward(ctx, do):
        q, k, v, o, lse = ctx.saved_tensors
        dq, dk, dv = attention_backward(do, q, k, v, o, lse, ctx.causal, ctx.scale, kv_lens=ctx.kv_lens)
        return dq, dk, dv, None, None, None


def flash_attention(q, k, v, causal: bool = True, scale: float | None = None, kv_lens=None):
    """Differentiable attention on [B, S, H, D] tensors.  CUDA: tiled flash kernels; CPU: reference math.
    `kv_lens` ([B] integers): number of real keys per batch entry (key-padding mask given as lengths)."""
    scale = 1.0 / math.sqrt(q.shape[-1]) if scale is None else scale
    if not q.is_cuda:
        return attention_reference(q, k, v, causal, scale, kv_lens)
    if kv_lens is not None:
        kv_lens = kv_lens.to(device=q.device, dtype=torch.int32).contiguous()
    D = q.shape[-1]
    in_dtype = q.dtype
    if in_dtype != torch.bfloat16:
        q, k, v = q.bfloat16(), k.bfloat16(), v.bfloat16()
    if D not in (64, 128):
        # The kernels take head dimensions 64 and 128.  Zero columns change neither QK^T nor the kept
        # columns of PV, so other sizes run padded (the scale stays that of the true head dimension).
        if D > 128:
            raise ValueError(f"flash_attention: head dimension {D} > 128 is not supported")
        Dp = 64 if D < 64 else 128
        pad = lambda t: torch.nn.functional.pad(t, (0, Dp - D))
        o = _FlashFn.apply(pad(q), pad(k), pad(v), causal, scale, kv_lens)[..., :D]
    else:
        q, k, v = (t if t.stride(3) == 1 else t.contiguous() for t in (q, k, v))
        o = _FlashFn.apply(q, k, v, causal, scale, kv_lens)
    return o if in_dtype == torch.bfloat16 else o.to(in_dtype)
