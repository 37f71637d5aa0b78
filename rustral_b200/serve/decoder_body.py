"""The layer bodies that the serving runner executes, one class per family of decoders.

A body knows a model's mathematics only: embedding, one layer, output head, and what each layer stores in the cache.  Which
rows a step holds, where their keys and values go, which kernels attend for which rows, and graph capture belong to the
runner (serve.model_runner), so every body gets prefill, chunked prefill, mixed batches and graphed decoding from it.

`embed` returns the stream that `layer` takes and returns; `head` turns selected rows of it into logits.  `depth` is the number of
layers that run (and have a cache each): a layer that is passed through several times counts as often.
"""
from __future__ import annotations

import math

import torch

from .. import ops
from ..models.layered import AttentionSpec, DenseSpec, LatentSpec, ParallelSpec, RetentionSpec, up8
from ..ops import latent as latent_ops
from ..ops import moe as moe_ops
from ..ops import norm as norm_ops
from ..ops import paged as paged_ops
from ..ops import recurrent as rc_ops
from ..ops import rotary as rope_ops
from ..ops.attention import ScoreRule, distance_slopes
from ..ops.heads import head_prep_, row_prep_
from ..ops.matmul import gemm
from .kv_cache import CacheLayer
from .weights import latent_columns, mixer_columns, packed_columns


class GPTBody:
    """GPT-2 style and Llama style decoders (pre-norm, residual stream in the activation dtype)."""

    def __init__(self, runner):
        self.r, self.cfg = runner, runner.cfg
        self.rms = self.cfg.arch == "llama"
        self.scale = 1.0 / math.sqrt(self.cfg.head_dim)
        self.depth = self.cfg.n_layer

    def cache_layers(self) -> list:
        return None                                   # uniform: the cache's num_layers / num_kv_heads / head_dim form

    def _norm(self, x, name):
        P, rms = self.r.params, self.rms
        y, _, _ = norm_ops.norm_forward(x, P.w(name + ".weight"), None if rms else P.w(name + ".bias"), self.cfg.norm_eps, rms)
        return y

    def _row_parallel(self, a, w, bias, residual):
        """a @ w^T (+ bias) + residual; with tensor parallelism the partial products are summed over the ranks."""
        tp = self.r.tp
        if tp is None:
            return gemm(a, w, bias=bias, residual=residual)
        rows = a.shape[0]
        gemm(a, w, out=tp.staging(rows, w.shape[0]))
        return tp.all_reduce(rows, w.shape[0], residual=residual)

    def embed(self, sb):
        P, cfg = self.r.params, self.cfg
        x = ops.embedding_forward(sb.ids, P.w("tok_embed.embed"))
        if cfg.arch == "gpt2":
            x = ops.binary("add", x, ops.gather_rows(P.w("pos_embed.embed"), sb.pos))
        return x

    def layer(self, l, x, sb):
        P, r, rms = self.r.params, self.r, self.rms
        H, Hk, D = r.n_head, r.n_kv_head, self.cfg.head_dim
        p = f"layers.{l}."
        h = self._norm(x, p + "ln1")
        qkv = gemm(h, P.w(p + "attn.wqkv.weight"), bias=None if rms else P.w(p + "attn.wqkv.bias"))
        if rms:
            rope_ops.rope_(qkv, H + Hk, D, positions=sb.pos, theta=self.cfg.rope_theta)
        k2, v2 = qkv[:, H * D:(H + Hk) * D], qkv[:, (H + Hk) * D:]
        paged_ops.kv_append(k2, v2, r.cache.k[l], r.cache.v[l], sb.slots)
        a = r.attend(l, qkv[:, :H * D], k2, v2, sb, self.scale)
        x = self._row_parallel(a, P.w(p + "attn.wo.weight"), None if rms else P.w(p + "attn.wo.bias"), x)
        h = self._norm(x, p + "ln2")
        if rms:
            gu = gemm(h, P.w(p + "ffn.gate_up.weight"))
            return self._row_parallel(rope_ops.swiglu_forward(gu), P.w(p + "ffn.down.weight"), None, x)
        h = gemm(h, P.w(p + "ffn.fc1.weight"), bias=P.w(p + "ffn.fc1.bias"), act="gelu")
        return gemm(h, P.w(p + "ffn.fc2.weight"), bias=P.w(p + "ffn.fc2.bias"), residual=x)

    def head(self, x, rows):
        P, cfg, tp = self.r.params, self.cfg, self.r.tp
        if rows is not None:
            x = x.index_select(0, rows)
        xf = self._norm(x.contiguous(), "final_norm")
        if tp is not None:
            w = P.w("head.weight")
            gemm(xf, w, out=tp.staging(xf.shape[0], w.shape[0]))
            return tp.all_gather_cols(xf.shape[0], w.shape[0])
        return gemm(xf, P.w("tok_embed.embed" if cfg.tie_embeddings else "head.weight"))


class Stream:
    """Residual stream of a layered decoder: `x` fp32, `h` its copy in the activation dtype (the operand of the next
    products; `x` itself in 32-bit), `v_first` the value columns of the first layer that mixes values, `pair` the copies of the
    stream and of the embedding side by side that a pass through repeated layers starts from, `kv` the step's keys and values of
    layers whose cache others use."""
    __slots__ = ("x", "h", "v_first", "pair", "kv")

    def __init__(self, x, h):
        self.x, self.h, self.v_first, self.pair, self.kv = x, h, None, None, {}


class LayeredBody:
    """Layered decoders (models.layered): sublayers read the stream itself, the norm sits on their output.

    Per layer: one packed projection; head norms + value mixing + cache append (one kernel); attention with its score rule
    and output gate; output projection; norm + residual add; router; experts as grouped products; shared expert; then
    combine + norm + residual add (one kernel)."""

    def __init__(self, runner):
        self.r, self.cfg = runner, runner.cfg
        if runner.tp is not None:
            raise ValueError("tensor-parallel serving covers the llama family")
        self.depth = self.cfg.n_layer
        slopes = {}
        self.rules = []
        for s in self.cfg.layers:
            a = s.mixer
            if a.heads not in slopes:
                slopes[a.heads] = distance_slopes(a.heads, runner.device)
            self.rules.append(ScoreRule(softcap=a.softcap, slopes=slopes[a.heads], chunk=a.chunk))

    def cache_layers(self) -> list:
        return [CacheLayer(s.mixer.kv_heads, s.mixer.dim, s.mixer.vdim) for s in self.cfg.layers]

    def embed(self, sb):
        return Stream(*ops.embedding_residual(sb.ids, self.r.params.w("embed")))

    def _add_norm(self, st, y, name, **kw):
        """x += norm(y), h = x in the activation dtype."""
        P = self.r.params
        norm_ops.residual_norm(y, P.w(name), P.w(name + ".b"), self.cfg.norm_eps, x=st.x,
                               h=None if st.h is st.x else st.h, **kw)

    def layer(self, l, st, sb):
        r, P, s = self.r, self.r.params, self.cfg.layers[l]
        a, p = s.mixer, f"l{l}."
        H, G, dk, dv = a.heads, a.kv_heads, a.dim, a.vdim
        z = gemm(st.h, P.w(p + "attn.in"))
        ov = (H + G) * dk
        k2, v2, gate = z[:, H * dk:ov], z[:, ov:ov + G * dv], z[:, ov + G * dv:]
        mixed = a.v_mix and l != self.cfg.first_mix
        head_prep_(z, H, G, dk, dv, q_gamma=P.w(p + "attn.q_norm"), k_gamma=P.w(p + "attn.k_norm"), eps=self.cfg.norm_eps,
                   v_first=st.v_first if mixed else None, mix=P.w(p + "attn.mix") if mixed else None,
                   k_cache=r.cache.k[l], v_cache=r.cache.v[l], slots=sb.slots)
        if l == self.cfg.first_mix:
            st.v_first = v2                            # a view: this layer's projection buffer stays alive
        o = r.attend(l, z[:, :H * dk], k2, v2, sb, a.scale, self.rules[l], gate)
        self._add_norm(st, gemm(o, P.w(p + "attn.out"), out_dtype=torch.float32), p + "norm1")
        if s.mlp is not None:
            self._experts(st, s.mlp, p)
        return st

    def _experts(self, st, m, p):
        P, h = self.r.params, st.h
        logits = gemm(h, P.w(p + "moe.router"), out_dtype=torch.float32)
        idx, w = moe_ops.route_groups(logits, m.top, m.groups, m.keep)
        pl = moe_ops.plan(idx, m.experts)
        gu = moe_ops.grouped_gemm(moe_ops.scatter_tokens(h, pl), P.w(p + "moe.w1"), pl)
        y = moe_ops.grouped_gemm(moe_ops.swiglu_rows(gu, pl), P.w(p + "moe.w2"), pl)
        shared = None
        if m.shared_ff:
            shared = gemm(moe_ops.swiglu_rows(gemm(h, P.w(p + "shared.in"))), P.w(p + "shared.out"))
        self._add_norm(st, y, p + "norm2", routed=(pl.slot_pos, w), add=shared)

    def head(self, st, rows):
        P, cfg = self.r.params, self.cfg
        x = st.x if rows is None else ops.gather_rows(st.x, rows)
        h = norm_ops.residual_norm(x, P.w("final.norm"), P.w("final.norm.b"), cfg.norm_eps, h=torch.empty_like(x, dtype=self.r.dtype))
        logits = gemm(h, P.w("head"), out_dtype=torch.float32)
        return ops.scale_softcap_(logits, cfg.logit_scale, cfg.logit_softcap)


class ParallelBody:
    """Layered decoders with one norm in front of a layer and mixer and feed-forward side by side behind it (Vafodra).

    Per layer: one packed projection of everything that reads the norm's output, and a narrow one whose results stay fp32 (step
    sizes, decays, per-head gates); the mixers; act(gate) * up; output projections (mixer and feed-forward as one product where
    their sum needs no norm); then norms of the mixer's outputs, residual add and the next layer's norm in one kernel."""

    def __init__(self, runner):
        self.r, self.cfg = runner, runner.cfg
        if runner.tp is not None:
            raise ValueError("tensor-parallel serving covers the llama family")
        self.depth = self.cfg.n_layer
        self.columns = [packed_columns(s) for s in self.cfg.layers]
        self.prefix = [f"l{self.cfg.owner(i)}." for i in range(self.cfg.n_layer)]
        slopes = {}
        self.rules = []
        for s in self.cfg.layers:
            a = s.mixer.left if isinstance(s.mixer, ParallelSpec) else None
            if a is not None and a.distance_bias and a.heads not in slopes:
                slopes[a.heads] = distance_slopes(a.heads, runner.device)
            self.rules.append(None if a is None else ScoreRule(a.softcap, slopes.get(a.heads), a.chunk, a.window, a.keep_first, a.sink))

    def cache_layers(self) -> list:
        out = []
        for s in self.cfg.layers:
            m = s.mixer
            if isinstance(m, ParallelSpec):
                a, r = m.left, m.right
                out.append(CacheLayer(a.kv_heads, a.dim, a.vdim, (("conv", (r.conv - 1, r.channels), None),
                                                                  ("state", (r.heads, r.state, rc_ops.up4(r.vdim)), torch.float32))))
            else:
                out.append(CacheLayer(state=(("conv", (m.conv - 1, m.channels), None),
                                             ("state", (m.heads, m.dim, rc_ops.up4(m.vdim)), torch.float32))))
        return out

    def _norm(self, name):
        P = self.r.params
        return P.w(name), P.w(name + ".b"), P.w(name + ".alpha")

    def _update(self, st, l, **sources):
        """x += residual_mult * (...), then the norm in front of layer l + 1 (the head takes its norm over the wanted rows)."""
        dyt = h = None
        if l + 1 < self.cfg.n_layer:
            dyt = self._norm(self.prefix[l + 1] + "norm1")
            h = torch.empty(st.x.shape, dtype=self.r.dtype, device=st.x.device)
        if sources or dyt is not None:
            norm_ops.stream_update(st.x, mult=self.cfg.residual_mult, eps=self.cfg.norm_eps, dyt=dyt, h=h, **sources)
        st.h = h
        return st

    def embed(self, sb):
        x, _ = ops.embedding_residual(sb.ids, self.r.params.w("embed"), self.cfg.embed_scale, want_h=False)
        return self._update(Stream(x, None), -1)

    def layer(self, l, st, sb):
        P, p, s = self.r.params, self.prefix[l], self.cfg.layers[l]
        cols, gates = self.columns[l]
        z = gemm(st.h, P.w(p + "in"))
        small = gemm(st.h, P.w(p + "gates"), out_dtype=torch.float32)
        run = self._parallel if isinstance(s.mixer, ParallelSpec) else self._delta
        return run(l, st, sb, s, p, lambda c: z[:, cols[c][0]:cols[c][0] + cols[c][1]], lambda c: small[:, gates[c][0]:gates[c][0] + gates[c][1]],
                   z)

    def _feed_forward(self, l, s, z, out=None):
        lo = self.columns[l][0]["gate"][0]
        return moe_ops.swiglu_rows(z[:, lo:lo + 2 * up8(s.mlp.ff)], act=s.mlp.act, out=out)

    def _parallel(self, l, st, sb, s, p, col, gate, z):
        r, P, cfg = self.r, self.r.params, self.cfg
        a, m = s.mixer.left, s.mixer.right
        k2, v2 = col("k"), col("v")
        head_prep_(z, a.heads, a.kv_heads, a.dim, a.vdim, k_cache=r.cache.k[l], v_cache=r.cache.v[l], slots=sb.slots)
        o = r.attend(l, col("q"), k2, v2, sb, a.scale, self.rules[l], head_gate=gate("g"))
        state = r.cache.state[l]
        xbc = rc_ops.short_conv(col("conv"), P.w(p + "conv"), P.w(p + "conv.b"), state["conv"], sb.segments)
        y = rc_ops.state_space(xbc, gate("dt"), dt_bias=P.w(p + "dt_bias"), a_log=P.w(p + "A_log"), D=P.w(p + "D"), state=state["state"],
                               heads=m.heads, groups=m.groups, vdim=m.vdim, n=m.state, seg=sb.segments)
        y = rc_ops.gated_norm(y, col("z"), P.w(p + "norm"), m.norm_groups, cfg.norm_eps, gate_first=True, out=y)
        out = dict(a=gemm(o, P.w(p + "left.o")), wa=P.w(p + "left.out"),
                   b=gemm(y, P.w(p + "right.o")), wb=P.w(p + "right.out"), normed=0.5)
        if s.mlp is not None:
            out["c"] = gemm(self._feed_forward(l, s, z), P.w(p + "down"))
        return self._update(st, l, **out)

    def _delta(self, l, st, sb, s, p, col, gate, z):
        P, m = self.r.params, s.mixer
        state = self.r.cache.state[l]
        n, w_out = m.heads * m.vdim, P.w(p + "out")
        qkv = rc_ops.short_conv(z[:, :m.channels], P.w(p + "conv"), None, state["conv"], sb.segments)
        joined = torch.empty((sb.rows, w_out.shape[1]), dtype=z.dtype, device=z.device)      # mixer output | feed-forward
        if up8(n) != n:
            joined[:, n:up8(n)] = 0
        o = rc_ops.delta_rule(qkv, gate("a"), gate("b"), dt_bias=P.w(p + "dt_bias"), a_log=P.w(p + "A_log"), state=state["state"],
                              heads=m.heads, kv_heads=m.kv_heads, dk=m.dim, dv=m.vdim, seg=sb.segments, out=joined[:, :n])
        rc_ops.gated_norm(o, col("z"), P.w(p + "norm"), m.heads, self.cfg.norm_eps, gate_first=False, out=o)
        if s.mlp is not None:
            self._feed_forward(l, s, z, out=joined[:, up8(n):])
        return self._update(st, l, c=gemm(joined, w_out))

    def head(self, st, rows):
        P = self.r.params
        x = st.x if rows is None else ops.gather_rows(st.x, rows)
        h = norm_ops.stream_update(x, dyt=self._norm("final.norm"), h=torch.empty(x.shape, dtype=self.r.dtype, device=x.device))
        logits = gemm(h, P.w("head"), out_dtype=torch.float32)
        if self.cfg.logit_scale != 1.0 or self.cfg.logit_softcap:
            ops.scale_softcap_(logits, self.cfg.logit_scale, self.cfg.logit_softcap)
        return logits


def _rotation_frequencies(rots, device) -> dict:
    """{rotary positions: angle per position of every pair (fp64)} of those that occur."""
    return {rot: torch.tensor(rot.frequencies(), dtype=torch.float64).to(device) for rot in rots if rot is not None}


def _rotation(sb, rot, freqs):
    """The step's cosines and sines for `rot` (None: no rotation)."""
    return None if rot is None or rot.dims == 0 else sb.rotation(rot, freqs[rot])


def _experts(P, h, m, p):
    """Routed feed-forward `m` (models.layered.MoESpec) over rows h: (expert rows, (their places, weights or None)) for the sum that
    ops.norm.residual_norm takes."""
    logits = gemm(h, P.w(p + "moe.router"), out_dtype=torch.float32)
    if m.score == "sigmoid":
        idx, w = moe_ops.route_sigmoid(logits, m.top, m.groups, m.keep, P.w(p + "moe.correction") if m.correction else None,
                                       m.group_best, m.renorm)
    else:
        idx, w = moe_ops.route_groups(logits, m.top, m.groups, m.keep, m.renorm)
    pl = moe_ops.plan(idx, m.experts)
    gu = moe_ops.grouped_gemm(moe_ops.scatter_tokens(h, pl), P.w(p + "moe.w1"), pl)
    at_input = m.weigh == "input"
    y = moe_ops.grouped_gemm(moe_ops.swiglu_rows(gu, pl, m.act, limit=m.limit, weights=w if at_input else None), P.w(p + "moe.w2"), pl)
    return y, (pl.slot_pos, None if at_input else w)


class SandwichBody:
    """Layered decoders with a norm in front of every sublayer and one on its output (Bikilix); some layers can run several times.

    Per layer: one packed projection of everything that reads the first norm; attention (head rotation + cache append in one kernel) or
    latent attention; output projection; then its norm, residual add and the norm in front of the feed-forward in one kernel; dense or
    routed feed-forward; its norm (with the experts' combine), residual add and the next layer's norm in one kernel.  In front of a
    pass the stream becomes a product of itself and the embedding: both are kept side by side as the product's operand."""

    def __init__(self, runner):
        self.r, self.cfg = runner, runner.cfg
        if runner.tp is not None:
            raise ValueError("tensor-parallel serving covers the llama family")
        self.runs = self.cfg.runs
        self.depth = len(self.runs)
        self.freqs = _rotation_frequencies([s.mixer.rot for s in self.cfg.layers], runner.device)
        self.columns = [latent_columns(s.mixer) if isinstance(s.mixer, LatentSpec) else None for s in self.cfg.layers]
        self.rules = [self._rule(s.mixer) for s in self.cfg.layers]

    @staticmethod
    def _rule(m):
        if isinstance(m, LatentSpec):
            return None
        rule = ScoreRule(softcap=m.softcap, chunk=m.chunk, window=m.window, keep_first=m.keep_first, sink=m.sink)
        return None if rule.plain and m.dim == m.vdim and m.dim in (64, 128) else rule      # plain attention of those sizes needs no rule

    def cache_layers(self) -> list:
        out = []
        for i, _ in self.runs:
            m = self.cfg.layers[i].mixer
            out.append(CacheLayer(1, m.cached, m.kv_rank, joint=True) if isinstance(m, LatentSpec) else CacheLayer(m.kv_heads, m.dim, m.vdim))
        return out

    def _start(self, st, run, y=None, name=None, **kw):
        """What stands between sublayers: x += norm(y) (none without `y`), then the operand that run number `run` starts from: its
        norm of the stream, or the stream's copy beside the embedding in front of a pass (the stream itself behind the last layer)."""
        P, eps = self.r.params, self.cfg.norm_eps
        i, opens = self.runs[run] if run < self.depth else (None, None)
        gamma = P.w(f"l{i}.norm1") if i is not None else None
        if opens is not None:
            left = st.pair[:, :self.cfg.d_model]
            if y is not None:
                norm_ops.residual_norm(y, P.w(name), None, eps, True, x=st.x, h=left, **kw)
            st.x = gemm(st.pair, P.w("loop.in"), bias=P.w("loop.step")[opens], out_dtype=torch.float32)
            y = None
        if i is None:
            norm_ops.residual_norm(y, P.w(name), None, eps, True, x=st.x, **kw)
        elif y is None:
            st.h = norm_ops.residual_norm(st.x, gamma, None, eps, True, h=torch.empty_like(st.x, dtype=self.r.dtype))
        else:
            norm_ops.residual_norm(y, P.w(name), None, eps, True, x=st.x, h=st.h, next_gamma=gamma, **kw)
        return st

    def embed(self, sb):
        P, d, scale = self.r.params, self.cfg.d_model, self.cfg.embed_scale
        if self.cfg.loop is None:
            st = Stream(ops.embedding_residual(sb.ids, P.w("embed"), scale, want_h=False)[0], None)
        else:
            pair = torch.empty((sb.rows, 2 * d), dtype=self.r.dtype, device=self.r.device)
            x, _ = ops.embedding_residual(sb.ids, P.w("embed"), scale, h=pair[:, d:])
            st = Stream(x, None)
            st.pair = pair
            if self.runs[0][1] is not None:                       # the first pass starts from the embedding twice
                pair[:, :d] = pair[:, d:]
        return self._start(st, 0)

    def layer(self, run, st, sb):
        r, P = self.r, self.r.params
        i, _ = self.runs[run]
        s, p = self.cfg.layers[i], f"l{i}."
        o = (self._latent if isinstance(s.mixer, LatentSpec) else self._attention)(run, i, s.mixer, p, st.h, sb)
        y = gemm(o, P.w(p + "attn.out"), out_dtype=torch.float32)
        if s.mlp is None:
            return self._start(st, run + 1, y, p + "norm1b")
        norm_ops.residual_norm(y, P.w(p + "norm1b"), None, self.cfg.norm_eps, True, x=st.x, h=st.h, next_gamma=P.w(p + "norm2"))
        if isinstance(s.mlp, DenseSpec):
            y = gemm(gemm(st.h, P.w(p + "up"), act=s.mlp.act), P.w(p + "down"), out_dtype=torch.float32)
            return self._start(st, run + 1, y, p + "norm2b")
        y, routed = _experts(P, st.h, s.mlp, p)
        return self._start(st, run + 1, y, p + "norm2b", routed=routed)

    def _attention(self, run, i, a, p, h, sb):
        r, P = self.r, self.r.params
        H, G, dk, dv = a.heads, a.kv_heads, a.dim, a.vdim
        z = gemm(h, P.w(p + "attn.in"), bias=P.w(p + "attn.in.b") if a.bias else None)
        ov = (H + G) * dk
        head_prep_(z, H, G, dk, dv, k_cache=r.cache.k[run], v_cache=r.cache.v[run], slots=sb.slots, rot=_rotation(sb, a.rot, self.freqs))
        return r.attend(run, z[:, :H * dk], z[:, H * dk:ov], z[:, ov:], sb, a.scale, self.rules[i])

    def _latent(self, run, i, m, p, h, sb):
        r, P, cols = self.r, self.r.params, self.columns[i]
        z = gemm(h, P.w(p + "attn.in"))
        part = lambda c: z[:, cols[c][0]:cols[c][0] + cols[c][1]]
        table = _rotation(sb, m.rot, self.freqs)
        latent_ops.latent_prep_(z, cols["q"][0], m.q_rank, cols["kv"][0], m.kv_rank, m.rot_dim, q_gamma=P.w(p + "attn.q_norm"),
                                kv_gamma=P.w(p + "attn.kv_norm"), eps=self.cfg.norm_eps, table=table, cache=r.cache.k[run], slots=sb.slots)
        q = gemm(part("q"), P.w(p + "attn.uq"))
        return r.attend_latent(run, q, part("kv"), sb, m, P.w(p + "attn.ukv"), table, part("g") if "g" in cols else None)

    def head(self, st, rows):
        P, cfg = self.r.params, self.cfg
        x = st.x if rows is None else ops.gather_rows(st.x, rows)
        h = norm_ops.residual_norm(x, P.w("final.norm"), None, cfg.norm_eps, True, h=torch.empty_like(x, dtype=self.r.dtype))
        logits = gemm(h, P.w("head"), out_dtype=torch.float32)
        if cfg.logit_scale != 1.0 or cfg.logit_softcap:
            ops.scale_softcap_(logits, cfg.logit_scale, cfg.logit_softcap)
        return logits


class PreNormBody:
    """Layered decoders with a norm in front of every sublayer, whose output is added as it is (Seredra).

    Per layer: one packed projection of everything that reads the first norm; the mixer; one output projection; residual add and the norm
    in front of the feed-forward in one kernel; dense or routed feed-forward; residual add (with the experts' sum) and the next layer's
    norm in one kernel.  Mixers: attention (short convolution; norm over the whole projection, temperature and cache append in one kernel;
    an attention layer can use the cache of an earlier one), retention (the state-space recurrence with fixed decays), or attention whose
    values are its keys beside a selective scan (both write one buffer, which one product reads)."""

    def __init__(self, runner):
        self.r, self.cfg = runner, runner.cfg
        if runner.tp is not None:
            raise ValueError("tensor-parallel serving covers the llama family")
        self.depth = self.cfg.n_layer
        mixers = [s.mixer for s in self.cfg.layers]
        self.freqs = _rotation_frequencies([m.left.rot if isinstance(m, ParallelSpec) else m.rot for m in mixers], runner.device)
        self.columns = [None if isinstance(m, AttentionSpec) else mixer_columns(m) for m in mixers]
        self.rules = [self._rule(l, m) for l, m in enumerate(mixers)]
        self.lent = {m.kv_from for m in mixers if isinstance(m, AttentionSpec) and m.kv_from is not None}

    def _rule(self, l, m):
        if isinstance(m, RetentionSpec):
            return None
        P, a, scale = self.r.params, m, 1.0
        if isinstance(m, ParallelSpec):
            a, scale = m.left, m.scales[0]
        logs = dict(log_amount=P.w(f"l{l}.attn.r1"), log_rate=P.w(f"l{l}.attn.r2")) if a.log_bias else {}
        return ScoreRule(a.softcap, None, a.chunk, a.window, a.keep_first, a.sink, out_scale=scale, **logs)

    def cache_layers(self) -> list:
        out = []
        for s in self.cfg.layers:
            m = s.mixer
            if isinstance(m, RetentionSpec):
                out.append(CacheLayer(state=(("state", (m.heads, m.dim, rc_ops.up4(m.vdim)), torch.float32),)))
            elif isinstance(m, ParallelSpec):
                a, r = m.left, m.right
                out.append(CacheLayer(a.kv_heads, a.dim, a.vdim, (("conv", (r.conv - 1, r.inner), None),
                                                                  ("state", (r.inner, rc_ops.up4(r.state)), torch.float32))))
            else:
                own = m.heads * m.dim + (m.kv_heads * (m.dim + m.vdim) if m.kv_from is None else 0)
                out.append(CacheLayer(m.kv_heads, m.dim, m.vdim, (("conv", (m.conv - 1, own), None),) if m.conv else (), kv_of=m.kv_from))
        return out

    def _start(self, st, l, y=None, **kw):
        """x += y (none without `y`; `kw`: see ops.norm.residual_norm), then the norm in front of layer l (the head takes its norm over
        the wanted rows)."""
        return self._add(st, self.r.params.w(f"l{l}.norm1") if l < self.depth else None, y, **kw)

    def _add(self, st, gamma, y=None, **kw):
        eps = self.cfg.norm_eps
        if y is None:
            st.h = norm_ops.residual_norm(st.x, gamma, None, eps, True, h=torch.empty_like(st.x, dtype=self.r.dtype))
        else:
            norm_ops.residual_norm(y, None, None, eps, True, x=st.x, h=None if gamma is None else st.h, next_gamma=gamma, **kw)
        return st

    def embed(self, sb):
        x, _ = ops.embedding_residual(sb.ids, self.r.params.w("embed"), self.cfg.embed_scale, want_h=False)
        return self._start(Stream(x, None), 0)

    def layer(self, l, st, sb):
        P, s, p = self.r.params, self.cfg.layers[l], f"l{l}."
        m = s.mixer
        mix = self._attention if isinstance(m, AttentionSpec) else self._retention if isinstance(m, RetentionSpec) else self._parallel
        o = mix(l, m, p, st, sb)
        y = gemm(o, P.w(p + "attn.out"), bias=P.w(p + "attn.out.b") if getattr(m, "out_bias", False) else None, out_dtype=torch.float32)
        if s.mlp is None:
            return self._start(st, l + 1, y)
        self._add(st, P.w(p + "norm2"), y)
        if isinstance(s.mlp, DenseSpec):
            return self._start(st, l + 1, gemm(gemm(st.h, P.w(p + "up"), act=s.mlp.act), P.w(p + "down"), out_dtype=torch.float32))
        y, routed = _experts(P, st.h, s.mlp, p)
        return self._start(st, l + 1, y, routed=routed)

    def _attention(self, l, a, p, st, sb):
        r, P = self.r, self.r.params
        H, dk, dv, own = a.heads, a.dim, a.vdim, a.kv_from is None
        G = a.kv_heads if own else 0
        z = gemm(st.h, P.w(p + "attn.in"), bias=P.w(p + "attn.in.b") if a.bias else None)
        if a.conv:
            z = rc_ops.short_conv(z, P.w(p + "attn.conv"), None, r.cache.state[l]["conv"], sb.segments, silu=False)
        row_prep_(z, H, G, dk, dv, q_gamma=P.w(p + "attn.q_norm"), k_gamma=P.w(p + "attn.k_norm") if own else None, eps=self.cfg.norm_eps,
                  pos=sb.pos, temp_coef=a.temp_coef, temp_every=a.temp_every, k_cache=r.cache.k[l], v_cache=r.cache.v[l], slots=sb.slots)
        q, ov = z[:, :H * dk], (H + G) * dk
        kv = (z[:, H * dk:ov], z[:, ov:]) if own else st.kv[a.kv_from]
        if l in self.lent:
            st.kv[l] = kv                                  # views: this layer's projection buffer stays alive
        return r.attend(l, q, *kv, sb, a.scale, self.rules[l])

    def _retention(self, l, m, p, st, sb):
        P, cols, H = self.r.params, self.columns[l], m.heads
        z = gemm(st.h, P.w(p + "attn.in"))
        head_prep_(z, H, H, m.dim, m.dim, rot=_rotation(sb, m.rot, self.freqs), half=True, k_scale=m.dim ** -0.5, q_col=cols["q"][0],
                   k_col=cols["k"][0])
        o = rc_ops.state_space(z[:, :H * (m.vdim + 2 * m.dim)], decay=P.w(p + "attn.decay"), state=self.r.cache.state[l]["state"], heads=H,
                               groups=H, vdim=m.vdim, n=m.dim, seg=sb.segments)
        lo, n = cols["g"]
        return rc_ops.gated_norm(o, z[:, lo:lo + n], None, H, self.cfg.norm_eps, gate_first=False, out=o)

    def _parallel(self, l, m, p, st, sb):
        r, P, cols = self.r, self.r.params, self.columns[l]
        a, s = m.left, m.right
        w_in, (lo, n) = P.w(p + "attn.in"), cols["v"]
        z = torch.empty((sb.rows, up8(lo + n)), dtype=r.dtype, device=r.device)
        gemm(st.h, w_in, out=z[:, :cols["end"][0]])
        part = lambda c: z[:, cols[c][0]:cols[c][0] + cols[c][1]]
        head_prep_(z, a.heads, a.kv_heads, a.dim, a.vdim, q_gamma=P.w(p + "attn.q_norm"), k_gamma=P.w(p + "attn.k_norm"), eps=self.cfg.norm_eps,
                   rot=_rotation(sb, a.rot, self.freqs), half=True, k_cache=r.cache.k[l], v_cache=r.cache.v[l], slots=sb.slots, v_col=lo,
                   values_are_keys=True)
        n, state = a.heads * a.vdim, r.cache.state[l]
        joined = torch.empty((sb.rows, P.w(p + "attn.out").shape[1]), dtype=r.dtype, device=r.device)       # attention | scan
        for edge, room in ((n, up8(n)), (up8(n) + s.inner, joined.shape[1])):
            if edge != room:
                joined[:, edge:room] = 0
        r.attend(l, part("q"), part("k"), part("v"), sb, a.scale, self.rules[l], out=joined[:, :n])
        x = rc_ops.short_conv(part("conv"), P.w(p + "scan.conv"), P.w(p + "scan.conv.b"), state["conv"], sb.segments)
        low = gemm(x, P.w(p + "scan.x"))
        r8, ns = up8(s.dt_rank), s.state
        dt = gemm(low[:, :r8], P.w(p + "scan.dt"), out_dtype=torch.float32)
        rc_ops.selective_scan(x, dt, low[:, r8:r8 + ns], low[:, r8 + ns:r8 + 2 * ns], part("z"), A=P.w(p + "scan.A"), D=P.w(p + "scan.D"),
                              dt_bias=P.w(p + "scan.dt.b"), state=state["state"], seg=sb.segments, scale=m.scales[1],
                              out=joined[:, up8(n):up8(n) + s.inner])
        return joined

    def head(self, st, rows):
        P = self.r.params
        x = st.x if rows is None else ops.gather_rows(st.x, rows)
        h = norm_ops.residual_norm(x, P.w("final.norm"), None, self.cfg.norm_eps, True, h=torch.empty_like(x, dtype=self.r.dtype))
        logits = gemm(h, P.w("head"), out_dtype=torch.float32)
        if self.cfg.logit_scale != 1.0 or self.cfg.logit_softcap:
            ops.scale_softcap_(logits, self.cfg.logit_scale, self.cfg.logit_softcap)
        return logits
