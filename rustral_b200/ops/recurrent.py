"""Mixers that carry state from token to token, over batches of unequal segments: short causal convolution, Mamba-2 state-space
recurrence (with a fixed decay: retention), Mamba's selective scan, gated delta rule, and the gated norm behind them.

Every op takes a `Segments` table (which rows belong to which sequence, where its state lives, whether it has just begun),
reads and updates the state tensors in place, and treats a sequence's state as zero at position 0.
"""
from __future__ import annotations

import torch

from .. import _native as N

CONV_TILE = 16
MAX_STATE_ROWS = 256
UNIT_EPS = 1e-6

N.optional_sig("rb_short_conv", [N.C.POINTER(N.RbShortConvArgs), N.c_void_p])
N.optional_sig("rb_state_space_scan", [N.C.POINTER(N.RbStateSpaceArgs), N.c_void_p])
N.optional_sig("rb_delta_rule_scan", [N.C.POINTER(N.RbDeltaRuleArgs), N.c_void_p])
N.optional_sig("rb_gated_norm", [N.C.POINTER(N.RbGatedNormArgs), N.c_void_p])
N.optional_sig("rb_state_space_chunked", [N.C.POINTER(N.RbStateSpaceArgs), N.c_void_p, N.c_void_p, N.c_int, N.c_void_p])
N.optional_sig("rb_delta_rule_chunked", [N.C.POINTER(N.RbDeltaRuleArgs), N.c_void_p])
N.optional_sig("rb_delta_rule_scratch_bytes", [N.c_int, N.c_int, N.c_int], N.c_ll)
N._LAUNCHES["rb_delta_rule_chunked"] = 2

CHUNK = 64                                            # tokens per step of the chunked kernels


class Segments:
    """Rows of a batch as segments, each the next tokens of one sequence.

    `table`: int32 [n, 4] on the device: first row, number of rows, state slot, position of the first row.  `rows`: the same as
    a list of tuples on the host, or None where only the device knows them (a captured decode step): then every segment is one
    row."""

    def __init__(self, table: torch.Tensor, rows: list | None):
        self.table, self.rows = table, rows
        self.n = table.shape[0]
        self._tiles: dict = {}
        self._split = None

    @classmethod
    def of(cls, rows: list, device) -> "Segments":
        return cls(torch.tensor(rows, dtype=torch.int32).view(-1, 4).to(device), rows)

    @property
    def single(self) -> bool:
        """Every segment is one row (a decode step)."""
        return self.rows is None or all(r[1] == 1 for r in self.rows)

    def split(self) -> tuple:
        """(segments of several rows, segments of one row), either None when there are none."""
        if self._split is None:
            if self.single:
                self._split = (None, self)
            else:
                many = [i for i, r in enumerate(self.rows) if r[1] > 1]
                one = [i for i, r in enumerate(self.rows) if r[1] <= 1]
                part = lambda idx: Segments(self.table[torch.tensor(idx, device=self.table.device)], [self.rows[i] for i in idx])
                self._split = (self if not one else part(many), part(one) if one else None)
        return self._split

    def tiles(self, size: int) -> torch.Tensor:
        """int32 [tiles, 2]: (segment, first row inside it) of pieces of at most `size` rows."""
        if size not in self._tiles:
            if self.single:
                if 1 not in self._tiles:
                    t = torch.zeros((self.n, 2), dtype=torch.int32, device=self.table.device)
                    t[:, 0] = torch.arange(self.n, dtype=torch.int32, device=self.table.device)
                    self._tiles[1] = t
                self._tiles[size] = self._tiles[1]
            else:
                pairs = [(i, o) for i, r in enumerate(self.rows) for o in range(0, r[1], size)]
                self._tiles[size] = torch.tensor(pairs, dtype=torch.int32).to(self.table.device)
        return self._tiles[size]

    def host(self) -> list:
        return self.rows if self.rows is not None else [tuple(r) for r in self.table.tolist()]


def up4(n: int) -> int:
    return (n + 3) // 4 * 4


def _check(t, dtype, what):
    if t.dtype != dtype or t.stride(-1) != 1:
        raise TypeError(f"{what}: {dtype} with a contiguous last dimension is required")


def short_conv(x, w, bias, state, seg: Segments, silu: bool = True, out=None):
    """out[t] = act(bias + sum_i w[:, i] * x[t - (taps - 1) + i]) per sequence.  x [rows, channels] (row-strided views allowed),
    w fp32 [channels, taps], bias fp32 [channels] or None, state [slots, taps - 1, channels] in the dtype of x."""
    rows, C = x.shape
    taps = w.shape[1]
    out = out if out is not None else torch.empty((rows, C), dtype=x.dtype, device=x.device)
    if not x.is_cuda:
        for first, n, slot, start in seg.host():
            past = state[slot].float() if start > 0 else torch.zeros(taps - 1, C)
            full = torch.cat([past, x[first:first + n].float()])
            y = sum(w[:, i].float() * full[i:i + n] for i in range(taps))
            if bias is not None:
                y = y + bias.float()
            out[first:first + n] = (y * torch.sigmoid(y) if silu else y).to(out.dtype)
            if taps > 1:
                state[slot] = full[n:].to(state.dtype)
        return out
    _check(w, torch.float32, "short_conv")
    a = N.RbShortConvArgs()
    tiles = seg.tiles(CONV_TILE)
    a.x, a.ld_x, a.out, a.ld_o = x.data_ptr(), x.stride(0), out.data_ptr(), out.stride(0)
    a.state, a.num_slots = state.data_ptr(), state.shape[0]
    a.w, a.bias, a.segments, a.tiles, a.num_tiles = w.data_ptr(), N.ptr(bias), seg.table.data_ptr(), tiles.data_ptr(), tiles.shape[0]
    a.channels, a.taps, a.f32, a.silu = C, taps, int(x.dtype == torch.float32), int(silu)
    N.check(N.kernels().rb_short_conv(a, N.stream_ptr()), "rb_short_conv")
    return out


def _softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def _chunked(x, rows: int, a: int, b: int) -> bool:
    """Whether the tensor-core kernels take prompts of these operands: `rows` state rows, head sizes a and b."""
    return x.dtype == torch.bfloat16 and rows <= 128 and a % 8 == 0 and b % 8 == 0 and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0


def _span(seg: Segments, ctas_per_span: int, slots: int = 148) -> int:
    """Rows per span of the chunked state-space kernel: the power of two for which the spans that run side by side cost least
    (rounds of `slots` CTAs, and about half of that again for the first pass where segments have several spans)."""
    lens = [r[1] for r in seg.rows]
    best, span = None, 0
    size = 256
    while True:
        spans = sum(-(-n // size) for n in lens)
        rows = min(size, max(lens))
        cost = -(-spans * ctas_per_span // slots) * (rows + 256.0)
        if spans > len(lens):
            cost += 0.5 * -(-(spans - len(lens)) * ctas_per_span // slots) * (rows + 256.0)
        if best is None or cost < best:
            best, span = cost, size
        if size >= max(lens):
            return span
        size *= 2


def state_space(xbc, dt_raw=None, *, dt_bias=None, a_log=None, D=None, state, heads: int, groups: int, vdim: int, n: int, seg: Segments,
                decay=None, out=None):
    """Mamba-2 recurrence, or with `decay` (fp32 [heads]; dt_raw, dt_bias and a_log None) one whose decays are fixed and whose step sizes
    are 1.  xbc [rows, heads * vdim + 2 * groups * n] = x | B | C behind the convolution; dt_raw fp32
    [rows, heads]; dt_bias, a_log, D fp32 [heads] (D None: 0); state fp32 [slots, heads, n, up4(vdim)].  Returns y [rows, heads * vdim]."""
    rows = xbc.shape[0]
    inner = heads * vdim
    out = out if out is not None else torch.empty((rows, inner), dtype=xbc.dtype, device=xbc.device)
    if not xbc.is_cuda:
        per = heads // groups
        x = xbc[:, :inner].float().view(rows, heads, vdim)
        B = xbc[:, inner:inner + groups * n].float().view(rows, groups, n).repeat_interleave(per, 1)
        C = xbc[:, inner + groups * n:inner + 2 * groups * n].float().view(rows, groups, n).repeat_interleave(per, 1)
        if decay is None:
            dt = _softplus(dt_raw.float() + dt_bias)
            decay = torch.exp(-torch.exp(a_log) * dt)
        else:
            dt, decay = torch.ones(rows, heads), decay.float().expand(rows, heads)
        for first, m, slot, start in seg.host():
            S = state[slot, :, :, :vdim].clone() if start > 0 else torch.zeros(heads, n, vdim)
            for t in range(first, first + m):
                S = decay[t, :, None, None] * S + (dt[t, :, None] * B[t])[:, :, None] * x[t, :, None, :]
                y = torch.einsum("hnp,hn->hp", S, C[t])
                out[t] = (y if D is None else y + D[:, None] * x[t]).reshape(-1).to(out.dtype)
            state[slot, :, :, :vdim] = S
        return out
    if n > MAX_STATE_ROWS:
        raise ValueError(f"state_space: at most {MAX_STATE_ROWS} state rows per head")
    if (decay is None) == (dt_raw is None):
        raise ValueError("state_space: either step sizes or fixed decays")
    many, one = seg.split() if _chunked(xbc, n, n, vdim) and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0 else (None, seg)
    a = N.RbStateSpaceArgs()
    a.xbc, a.ld_xbc, a.y, a.ld_y = xbc.data_ptr(), xbc.stride(0), out.data_ptr(), out.stride(0)
    if decay is None:
        _check(dt_raw, torch.float32, "state_space")
        a.dt_raw, a.ld_dt, a.dt_bias, a.a_log = dt_raw.data_ptr(), dt_raw.stride(0), dt_bias.data_ptr(), a_log.data_ptr()
    else:
        _check(decay, torch.float32, "state_space")
        a.decay = decay.data_ptr()
    a.D, a.state, a.num_slots = N.ptr(D), state.data_ptr(), state.shape[0]
    a.heads, a.groups, a.p, a.n, a.f32 = heads, groups, vdim, n, int(xbc.dtype == torch.float32)
    if one is not None:
        a.segments, a.num_segments = one.table.data_ptr(), one.n
        N.check(N.kernels().rb_state_space_scan(a, N.stream_ptr()), "rb_state_space_scan")
    if many is not None:
        span = _span(many, heads * ((vdim + 63) // 64))
        tiles = many.tiles(span)
        a.segments, a.num_segments, a.tiles, a.num_tiles = many.table.data_ptr(), many.n, tiles.data_ptr(), tiles.shape[0]
        a.rows = rows
        states = decays = None
        if tiles.shape[0] > many.n:
            states = torch.empty((tiles.shape[0], heads, n, vdim), dtype=torch.float32, device=xbc.device)
            decays = torch.empty((tiles.shape[0], heads), dtype=torch.float32, device=xbc.device)
        N.check(N.kernels().rb_state_space_chunked(a, N.ptr(states), N.ptr(decays), span, N.stream_ptr()), "rb_state_space_chunked")
    return out


N.optional_sig("rb_selective_scan", [N.C.POINTER(N.RbSelectiveScanArgs), N.c_void_p])
MAX_CHANNEL_STATE = 256


def selective_scan(x, dt_raw, B, C, z, *, A, D, dt_bias, state, seg: Segments, scale: float = 1.0, out=None):
    """Mamba's recurrence.  Per channel c, with dt = softplus(dt_raw + dt_bias): S[c] <- exp(dt_c A[c]) S[c] + dt_c x_c B,
    y_c = S[c] . C + D_c x_c; out = scale * y * silu(z).  x, z [rows, inner], B, C [rows, n] (one dtype, row-strided views allowed; B and
    C with one pitch), dt_raw fp32 [rows, inner], A fp32 [inner, n] (negative), D, dt_bias fp32 [inner], state fp32 [slots, inner, up4(n)]."""
    rows, inner = x.shape
    n = A.shape[1]
    out = out if out is not None else torch.empty((rows, inner), dtype=x.dtype, device=x.device)
    if not x.is_cuda:
        dt = _softplus(dt_raw.float() + dt_bias)
        xf, zf = x.float(), z.float()
        for first, m, slot, start in seg.host():
            S = state[slot, :, :n].clone() if start > 0 else torch.zeros(inner, n)
            for t in range(first, first + m):
                S = torch.exp(dt[t, :, None] * A) * S + (dt[t] * xf[t])[:, None] * B[t].float()[None, :]
                y = S @ C[t].float() + D * xf[t]
                out[t] = (scale * y * (zf[t] * torch.sigmoid(zf[t]))).to(out.dtype)
            state[slot, :, :n] = S
        return out
    if n > MAX_CHANNEL_STATE:
        raise ValueError(f"selective_scan: at most {MAX_CHANNEL_STATE} numbers of state per channel")
    for t in (dt_raw, A, D, dt_bias, state):
        _check(t, torch.float32, "selective_scan")
    for t in (z, B, C):
        _check(t, x.dtype, "selective_scan")
    if B.stride(0) != C.stride(0) or not A.is_contiguous():
        raise ValueError("selective_scan: B and C have one pitch, and A is contiguous")
    a = N.RbSelectiveScanArgs()
    a.x, a.ld_x, a.z, a.ld_z, a.dt_raw, a.ld_dt = x.data_ptr(), x.stride(0), z.data_ptr(), z.stride(0), dt_raw.data_ptr(), dt_raw.stride(0)
    a.B, a.C, a.ld_bc, a.y, a.ld_y = B.data_ptr(), C.data_ptr(), B.stride(0), out.data_ptr(), out.stride(0)
    a.A, a.D, a.dt_bias, a.state, a.num_slots = A.data_ptr(), D.data_ptr(), dt_bias.data_ptr(), state.data_ptr(), state.shape[0]
    a.inner, a.n, a.f32, a.scale = inner, n, int(x.dtype == torch.float32), scale
    for part in seg.split():
        if part is not None:
            a.segments, a.num_segments, a.single = part.table.data_ptr(), part.n, int(part.single)
            N.check(N.kernels().rb_selective_scan(a, N.stream_ptr()), "rb_selective_scan")
    return out


def delta_rule(qkv, a_raw, b_raw, *, dt_bias, a_log, state, heads: int, kv_heads: int, dk: int, dv: int, seg: Segments, out=None):
    """Gated delta rule.  qkv [rows, 2 * kv_heads * dk + heads * dv] = q | k | v behind the convolution; a_raw, b_raw fp32
    [rows, heads] (same pitch); dt_bias, a_log fp32 [heads]; state fp32 [slots, heads, dk, up4(dv)].  Returns o
    [rows, heads * dv] (row-strided `out` allowed)."""
    rows = qkv.shape[0]
    out = out if out is not None else torch.empty((rows, heads * dv), dtype=qkv.dtype, device=qkv.device)
    if not qkv.is_cuda:
        per, nk = heads // kv_heads, kv_heads * dk
        unit = lambda t: t / torch.sqrt((t * t).sum(-1, keepdim=True) + UNIT_EPS)
        q = unit(qkv[:, :nk].float().view(rows, kv_heads, dk)).repeat_interleave(per, 1) * dk ** -0.5
        k = unit(qkv[:, nk:2 * nk].float().view(rows, kv_heads, dk)).repeat_interleave(per, 1)
        v = qkv[:, 2 * nk:2 * nk + heads * dv].float().view(rows, heads, dv)
        beta = torch.sigmoid(b_raw.float())
        decay = torch.exp(-torch.exp(a_log) * _softplus(a_raw.float() + dt_bias))
        for first, m, slot, start in seg.host():
            S = state[slot, :, :, :dv].clone() if start > 0 else torch.zeros(heads, dk, dv)
            for t in range(first, first + m):
                S = decay[t, :, None, None] * S
                u = beta[t, :, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
                S = S + k[t, :, :, None] * u[:, None, :]
                out[t] = torch.einsum("hkv,hk->hv", S, q[t]).reshape(-1).to(out.dtype)
            state[slot, :, :, :dv] = S
        return out
    if dk > MAX_STATE_ROWS:
        raise ValueError(f"delta_rule: key size at most {MAX_STATE_ROWS}")
    _check(a_raw, torch.float32, "delta_rule")
    _check(b_raw, torch.float32, "delta_rule")
    if a_raw.stride(0) != b_raw.stride(0):
        raise ValueError("delta_rule: a_raw and b_raw must have the same pitch")
    many, one = seg.split() if _chunked(qkv, dk, dk, dv) and out.stride(0) % 2 == 0 and out.data_ptr() % 4 == 0 else (None, seg)
    a = N.RbDeltaRuleArgs()
    a.qkv, a.ld_qkv, a.o, a.ld_o = qkv.data_ptr(), qkv.stride(0), out.data_ptr(), out.stride(0)
    a.a_raw, a.b_raw, a.ld_ab = a_raw.data_ptr(), b_raw.data_ptr(), a_raw.stride(0)
    a.dt_bias, a.a_log, a.state, a.num_slots = dt_bias.data_ptr(), a_log.data_ptr(), state.data_ptr(), state.shape[0]
    a.heads, a.kv_heads, a.dk, a.dv, a.f32 = heads, kv_heads, dk, dv, int(qkv.dtype == torch.float32)
    lib = N.kernels()
    if one is not None:
        a.segments, a.num_segments = one.table.data_ptr(), one.n
        N.check(lib.rb_delta_rule_scan(a, N.stream_ptr()), "rb_delta_rule_scan")
    if many is not None:
        tiles = many.tiles(CHUNK)
        scratch = torch.empty(lib.rb_delta_rule_scratch_bytes(tiles.shape[0], heads, dk), dtype=torch.uint8, device=qkv.device)
        a.segments, a.num_segments, a.tiles, a.num_tiles = many.table.data_ptr(), many.n, tiles.data_ptr(), tiles.shape[0]
        a.scratch, a.rows = scratch.data_ptr(), rows
        N.check(lib.rb_delta_rule_chunked(a, N.stream_ptr()), "rb_delta_rule_chunked")
    return out


def gated_norm(y, z, weight, parts: int, eps: float, gate_first: bool, out=None):
    """RMS norm of every one of `parts` equal parts of y's rows, gated with silu(z) before (gate_first) or behind the norm.
    weight fp32: one per column, or one part's, shared by all parts (None: no weight)."""
    rows, n = y.shape
    m = n // parts
    out = out if out is not None else torch.empty((rows, n), dtype=y.dtype, device=y.device)
    if not y.is_cuda:
        zf = z.float().view(rows, parts, m)
        g = zf * torch.sigmoid(zf)
        u = y.float().view(rows, parts, m)
        if gate_first:
            u = u * g
        u = u * torch.rsqrt((u * u).mean(-1, keepdim=True) + eps)
        if weight is not None:
            u = u * weight.view(-1, m)
        if not gate_first:
            u = u * g
        return out.copy_(u.reshape(rows, n))
    a = N.RbGatedNormArgs()
    a.y, a.ld_y, a.z, a.ld_z, a.out, a.ld_o = y.data_ptr(), y.stride(0), z.data_ptr(), z.stride(0), out.data_ptr(), out.stride(0)
    a.weight, a.weight_n = N.ptr(weight), m if weight is None else weight.numel()
    a.rows, a.parts, a.part_n, a.f32, a.gate_first, a.eps = rows, parts, m, int(y.dtype == torch.float32), int(gate_first), eps
    N.check(N.kernels().rb_gated_norm(a, N.stream_ptr()), "rb_gated_norm")
    return out
