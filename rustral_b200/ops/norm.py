"""LayerNorm / RMSNorm (bf16 activations, fp32 statistics) with explicit forward / backward entry points."""
from __future__ import annotations

import torch

from .. import _native as N

_scratch: dict = {}


def _partial_scratch(device, numel: int) -> torch.Tensor:
    """Grow-only fp32 scratch for the parameter-gradient partials, one per device and stream."""
    key = N.stream_key(device)
    buf = _scratch.get(key)
    if buf is None or buf.numel() < numel:
        buf = torch.empty(max(numel, 1 << 16), dtype=torch.float32, device=device)
        _scratch[key] = buf
    return buf


def norm_forward(x2: torch.Tensor, gamma: torch.Tensor, beta, eps: float, rms: bool, out=None, want_stats: bool = True):
    """x2: [rows, n].  Returns (y, mean, rstd); mean is None for RMSNorm, and both are None on a CUDA tensor when
    `want_stats` is False (inference: nothing will run backward)."""
    rows, n = x2.shape
    if not x2.is_cuda:
        xf = x2.float()
        if rms:
            mean = None
            rstd = torch.rsqrt((xf * xf).mean(-1) + eps)
            y = xf * rstd[:, None] * gamma.float()
        else:
            mean = xf.mean(-1)
            var = ((xf - mean[:, None]) ** 2).mean(-1)
            rstd = torch.rsqrt(var + eps)
            y = (xf - mean[:, None]) * rstd[:, None] * gamma.float()
            if beta is not None:
                y = y + beta.float()
        y = y.to(x2.dtype)
        if out is not None:
            out.copy_(y)
            y = out
        return y, mean, rstd
    if x2.dtype != torch.bfloat16 or gamma.dtype != torch.bfloat16:
        raise TypeError("norm: CUDA tensors must be bf16")
    y = out if out is not None else torch.empty((rows, n), dtype=x2.dtype, device=x2.device)
    mean = rstd = None
    if want_stats:
        if rms:
            rstd = torch.empty(rows, dtype=torch.float32, device=x2.device)
        else:
            mean, rstd = torch.empty((2, rows), dtype=torch.float32, device=x2.device).unbind(0)
    if rows == 0:
        return y, mean, rstd
    N.check(N.kernels().rb_norm_fwd(x2.data_ptr(), x2.stride(0), gamma.data_ptr(), N.ptr(beta), y.data_ptr(),
                                    y.stride(0), N.ptr(mean), N.ptr(rstd), rows, n, eps, int(rms),
                                    N.stream_ptr()), "rb_norm_fwd")
    return y, mean, rstd


def norm_backward(dy2, x2, gamma, mean, rstd, rms: bool, dres=None, dgamma=None, dbeta=None, accumulate=False,
                  dx_out=None):
    """Returns (dx, dgamma, dbeta); dgamma/dbeta are fp32.  `dres` (same shape as dx) is added into dx."""
    rows, n = x2.shape
    if not x2.is_cuda:
        xf, g = x2.float(), dy2.float()
        m = torch.zeros(rows) if rms else mean
        xhat = (xf - m[:, None]) * rstd[:, None]
        dg = (g * xhat).sum(0)
        db = None if rms else g.sum(0)
        gd = g * gamma.float()
        s1 = torch.zeros(rows, 1) if rms else gd.mean(-1, keepdim=True)
        s2 = (gd * xhat).mean(-1, keepdim=True)
        dx = rstd[:, None] * (gd - s1 - xhat * s2)
        if dres is not None:
            dx = dx + dres.float()
        dx = dx.to(x2.dtype)
        if dx_out is not None:
            dx_out.copy_(dx)
            dx = dx_out
        if dgamma is not None:
            dgamma.copy_(dgamma + dg if accumulate else dg)
            dg = dgamma
        if dbeta is not None and db is not None:
            dbeta.copy_(dbeta + db if accumulate else db)
            db = dbeta
        return dx, dg, db
    lib = N.kernels()
    nparts = lib.rb_norm_bwd_num_partials(rows, n)
    partial = _partial_scratch(x2.device, 2 * nparts * n)
    dx = dx_out if dx_out is not None else torch.empty_like(x2)
    if dgamma is None:
        dgamma = torch.empty(n, dtype=torch.float32, device=x2.device)
        accumulate = False
    if dbeta is None and not rms:
        dbeta = torch.empty(n, dtype=torch.float32, device=x2.device)
    N.check(lib.rb_norm_bwd(dy2.data_ptr(), dy2.stride(0), x2.data_ptr(), x2.stride(0), gamma.data_ptr(),
                            N.ptr(mean), rstd.data_ptr(), N.ptr(dres), dres.stride(0) if dres is not None else 0,
                            dx.data_ptr(), dx.stride(0), dgamma.data_ptr(), N.ptr(dbeta), partial.data_ptr(),
                            rows, n, int(rms), int(accumulate), N.stream_ptr()), "rb_norm_bwd")
    return dx, dgamma, dbeta


class _NormFn(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, gamma, beta, eps, rms):
        x2 = x.reshape(-1, x.shape[-1])
        if not x2.is_contiguous():
            x2 = x2.contiguous()
        y, mean, rstd = norm_forward(x2, gamma, beta, eps, rms)
        ctx.save_for_backward(x2, gamma, mean if mean is not None else rstd, rstd)
        ctx.rms = rms
        ctx.has_beta = beta is not None
        ctx.shape = x.shape
        return y.reshape(x.shape)

    @staticmethod
    def backward(ctx, dy):
        x2, gamma, mean, rstd = ctx.saved_tensors
        dy2 = dy.reshape(-1, dy.shape[-1])
        if not dy2.is_contiguous():
            dy2 = dy2.contiguous()
        dx, dg, db = norm_backward(dy2, x2, gamma, None if ctx.rms else mean, rstd, ctx.rms)
        return (dx.reshape(ctx.shape), dg.to(gamma.dtype), db.to(gamma.dtype) if (ctx.has_beta and db is not None) else None,
                None, None)


def _norm_inference(x, gamma, beta, eps, rms):
    x2 = x if x.dim() == 2 else x.reshape(-1, x.shape[-1])
    if not x2.is_contiguous():
        x2 = x2.contiguous()
    y = norm_forward(x2, gamma, beta, eps, rms, want_stats=False)[0]
    return y if x.dim() == 2 else y.reshape(x.shape)


def layer_norm(x, gamma, beta, eps: float = 1e-5):
    """Population variance, eps inside the square root (crates/nn/src/normalization.rs:87-158)."""
    if not N.wants_grad(x, gamma, beta):
        return _norm_inference(x, gamma, beta, eps, False)
    return _NormFn.apply(x, gamma, beta, eps, False)


def rms_norm(x, gamma, eps: float = 1e-5):
    if not N.wants_grad(x, gamma):
        return _norm_inference(x, gamma, None, eps, True)
    return _NormFn.apply(x, gamma, None, eps, True)


N.optional_sig("rb_residual_norm", [N.C.POINTER(N.RbResidualNormArgs), N.c_void_p])


def residual_norm(y, gamma, beta, eps: float, rms: bool = False, *, x=None, h=None, routed=None, add=None, next_gamma=None):
    """Norm of a sublayer's output added to a 32-bit residual stream.

    source row t = y[t], or with `routed` = (slot_pos int32 [T * k], weights fp32 [T, k]) the weighted sum of token t's
    expert rows of `y`; `add` (same dtype as y) is added to it.  With `x` (fp32 [T, n]): x += norm(source) in place and
    `h` receives a copy in its own dtype, or with `next_gamma` (dtype of gamma) rms(x) * next_gamma.  Without `x`: `h` receives
    norm(source).  `gamma` None: the source is added as it is (`next_gamma` is then fp32).  Expert weights None: all are 1.  Returns h
    (x when h is None)."""
    rows = x.shape[0] if x is not None else h.shape[0]
    n = y.shape[1]
    if not y.is_cuda:
        src = y.float()
        if routed is not None:
            slot_pos, w = routed
            src = src[slot_pos.long()].view(rows, -1, n)
            src = (src if w is None else src * w.float()[:, :, None]).sum(1)
        if add is not None:
            src = src + add.float()
        o = src if gamma is None else norm_forward(src, gamma, beta, eps, rms)[0].float()
        if x is not None:
            x += o
            o = x if next_gamma is None else norm_forward(x, next_gamma, None, eps, True)[0]
        if h is not None:
            h.copy_(o)
        return h if h is not None else x
    a = N.RbResidualNormArgs()
    a.y, a.ldy, a.y_f32 = y.data_ptr(), y.stride(0), int(y.dtype == torch.float32)
    if add is not None:
        if add.dtype != y.dtype:
            raise TypeError("residual_norm: `add` and `y` must have the same dtype")
        a.add, a.ld_add = add.data_ptr(), add.stride(0)
    if routed is not None:
        slot_pos, w = routed
        a.slot_pos, a.slot_w, a.k = slot_pos.data_ptr(), N.ptr(w), slot_pos.numel() // rows
    a.next_gamma = N.ptr(next_gamma)
    a.gamma, a.beta, a.param_f32 = N.ptr(gamma), N.ptr(beta), int(gamma is None or gamma.dtype == torch.float32)
    if x is not None:
        if x.dtype != torch.float32:
            raise TypeError("residual_norm: the residual stream is fp32")
        a.x, a.ldx = x.data_ptr(), x.stride(0)
    if h is not None:
        a.h, a.ldh, a.h_f32 = h.data_ptr(), h.stride(0), int(h.dtype == torch.float32)
    a.rows, a.n, a.rms, a.eps = rows, n, int(rms), eps
    N.check(N.kernels().rb_residual_norm(a, N.stream_ptr()), "rb_residual_norm")
    return h if h is not None else x


N.optional_sig("rb_stream_update", [N.C.POINTER(N.RbStreamUpdateArgs), N.c_void_p])


def stream_update(x, *, a=None, wa=None, b=None, wb=None, c=None, normed: float = 1.0, mult: float = 1.0, eps: float = 1e-5,
                  dyt=None, h=None):
    """x += mult * (normed * rms(a) * wa + normed * rms(b) * wb + c) on a 32-bit residual stream (in place; x is left as it is
    without a, b and c), then h = tanh(alpha x) * gamma + beta with dyt = (gamma fp32 [n], beta fp32 [n], alpha fp32 [1]).  a, b
    and c share their dtype.  Returns h, or x without `dyt`."""
    rows, n = x.shape
    src = [t for t in (a, b, c) if t is not None]
    if not x.is_cuda:
        v = torch.zeros_like(x)
        for t, w in ((a, wa), (b, wb)):
            if t is not None:
                tf = t.float()
                v += normed * tf * torch.rsqrt((tf * tf).mean(-1, keepdim=True) + eps) * w
        if c is not None:
            v += c.float()
        if src:
            x += mult * v
        if dyt is None:
            return x
        g, beta, alpha = dyt
        o = torch.tanh(alpha * x) * g + beta
        return o if h is None else h.copy_(o)
    if x.dtype != torch.float32 or len({t.dtype for t in src}) > 1:
        raise TypeError("stream_update: the residual stream is fp32 and its sources share a dtype")
    s = N.RbStreamUpdateArgs()
    s.x, s.ldx, s.rows, s.n, s.mult, s.normed, s.eps = x.data_ptr(), x.stride(0), rows, n, mult, normed, eps
    if a is not None:
        s.a, s.lda, s.wa = a.data_ptr(), a.stride(0), wa.data_ptr()
    if b is not None:
        s.b, s.ldb, s.wb = b.data_ptr(), b.stride(0), wb.data_ptr()
    if c is not None:
        s.c, s.ldc = c.data_ptr(), c.stride(0)
    s.y_f32 = int(bool(src) and src[0].dtype == torch.float32)
    if dyt is not None:
        g, beta, alpha = dyt
        h = h if h is not None else torch.empty_like(x)
        s.gamma, s.beta, s.alpha = g.data_ptr(), beta.data_ptr(), alpha.data_ptr()
        s.h, s.ldh, s.h_f32 = h.data_ptr(), h.stride(0), int(h.dtype == torch.float32)
    N.check(N.kernels().rb_stream_update(s, N.stream_ptr()), "rb_stream_update")
    return x if dyt is None else h
