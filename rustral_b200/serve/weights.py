"""Inference weights (bf16; layered decoders also fp32), optionally sharded for tensor parallelism, under the parameter names the
model runner uses.  Column-parallel matrices (QKV, gate/up, LM head) keep `1 / world` of their rows, row-parallel ones
(attention output, down projection) `1 / world` of their columns; norms and the embedding are replicated."""
from __future__ import annotations

import math
import zlib

import torch

from ..models.config import GPTConfig
from ..models.layered import AttentionSpec, DenseSpec, LatentSpec, ParallelSpec, RetentionSpec, up8


class InferenceWeights:
    def __init__(self, tensors: dict, dtype):
        self.tensors = tensors
        self.lowp = next(iter(tensors.values())).new_empty(0, dtype=dtype)   # dtype / device carrier

    def w(self, name: str) -> torch.Tensor:
        return self.tensors[name]

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.tensors.values())

    def load_state_dict(self, state: dict, cfg: GPTConfig) -> None:
        """Strict load of an UNSHARDED Llama-style checkpoint in the trainer's format (`FlatParams.state_dict`: fp32,
        vocabulary unpadded, attention projections under attn.wq / wk / wv): every expected key present, no extra
        key, shapes equal; nothing is written before all checks pass.  Tensor-parallel ranks load the full set and
        cut their shard with `shard_of`."""
        from ..core.errors import SerializationError, ShapeMismatch
        plan = {}                                         # checkpoint key -> (destination tensor, row slice)
        hd = cfg.head_dim
        q_end, k_end = cfg.n_head * hd, (cfg.n_head + cfg.n_kv_head) * hd
        for name, t in self.tensors.items():
            if ".attn.wqkv." in name:
                for nm, sl in (("wq", slice(0, q_end)), ("wk", slice(q_end, k_end)), ("wv", slice(k_end, t.shape[0]))):
                    plan[name.replace("wqkv", nm)] = (t, sl)
            elif name in ("tok_embed.embed", "head.weight"):
                plan[name] = (t, slice(0, cfg.vocab_size))
            else:
                plan[name] = (t, slice(0, t.shape[0]))
        missing = [k for k in plan if k not in state]
        extra = [k for k in state if k not in plan]
        if missing:
            raise SerializationError(f"missing keys: {missing}")
        if extra:
            raise SerializationError(f"unexpected keys: {extra}")
        for k, (t, sl) in plan.items():
            want = (sl.stop - sl.start, *t.shape[1:])
            if tuple(state[k].shape) != want:
                raise ShapeMismatch(want, state[k].shape, k)
        with torch.no_grad():
            for k, (t, sl) in plan.items():
                t[sl].copy_(state[k].to(t.device, t.dtype))

    # ------------------------------------------------------------------------------------------------ constructors
    @classmethod
    def random_llama(cls, cfg: GPTConfig, device, rank: int = 0, world: int = 1, seed: int = 0) -> "InferenceWeights":
        """Random-init Llama-style shard generated on the device (a full 8B model never exists on one GPU)."""
        if cfg.arch != "llama":
            raise ValueError("random_llama: llama-style configs only")
        dev = torch.device(device)
        dt = torch.bfloat16 if dev.type == "cuda" else torch.float32
        d, hd = cfg.d_model, cfg.head_dim
        hq, hk, f, v = cfg.n_head // world, cfg.n_kv_head // world, cfg.ffn_dim // world, cfg.vocab_padded // world

        def rnd(shape, name, shard, std):
            g = torch.Generator(device=dev).manual_seed((zlib.crc32(f"{seed}/{name}".encode()) & 0x7FFFFFFF) * 64 + shard)
            return torch.empty(shape, dtype=torch.float32, device=dev).normal_(0.0, std, generator=g).to(dt)

        t = {"tok_embed.embed": rnd((cfg.vocab_padded, d), "tok_embed", 0, cfg.init_std),
             "final_norm.weight": torch.ones(d, dtype=dt, device=dev),
             "head.weight": rnd((v, d), "head", rank, cfg.init_std)}
        s2 = cfg.init_std / math.sqrt(2 * cfg.n_layer)
        for l in range(cfg.n_layer):
            p = f"layers.{l}."
            t[p + "ln1.weight"] = torch.ones(d, dtype=dt, device=dev)
            t[p + "ln2.weight"] = torch.ones(d, dtype=dt, device=dev)
            t[p + "attn.wqkv.weight"] = rnd(((hq + 2 * hk) * hd, d), p + "wqkv", rank, cfg.init_std)
            t[p + "attn.wo.weight"] = rnd((d, hq * hd), p + "wo", rank, s2)
            t[p + "ffn.gate_up.weight"] = rnd((2 * f, d), p + "gate_up", rank, cfg.init_std)
            t[p + "ffn.down.weight"] = rnd((d, f), p + "down", rank, s2)
        return cls(t, dt)

    @classmethod
    def shard_of(cls, full, cfg: GPTConfig, rank: int, world: int) -> "InferenceWeights":
        """This rank's shard of a full Llama-style parameter set (`full.w(name)` gives the unsharded tensors)."""
        d, hd = cfg.d_model, cfg.head_dim
        H, Hk, F = cfg.n_head, cfg.n_kv_head, cfg.ffn_dim
        hq, hk, f, v = H // world, Hk // world, F // world, cfg.vocab_padded // world
        t = {"tok_embed.embed": full.w("tok_embed.embed"), "final_norm.weight": full.w("final_norm.weight"),
             "head.weight": full.w("head.weight")[rank * v:(rank + 1) * v].contiguous()}
        for l in range(cfg.n_layer):
            p = f"layers.{l}."
            t[p + "ln1.weight"], t[p + "ln2.weight"] = full.w(p + "ln1.weight"), full.w(p + "ln2.weight")
            wqkv = full.w(p + "attn.wqkv.weight")
            q = wqkv[:H * hd][rank * hq * hd:(rank + 1) * hq * hd]
            k = wqkv[H * hd:(H + Hk) * hd][rank * hk * hd:(rank + 1) * hk * hd]
            vv = wqkv[(H + Hk) * hd:][rank * hk * hd:(rank + 1) * hk * hd]
            t[p + "attn.wqkv.weight"] = torch.cat([q, k, vv], 0).contiguous()
            t[p + "attn.wo.weight"] = full.w(p + "attn.wo.weight")[:, rank * hq * hd:(rank + 1) * hq * hd].contiguous()
            gu = full.w(p + "ffn.gate_up.weight")
            t[p + "ffn.gate_up.weight"] = torch.cat([gu[:F][rank * f:(rank + 1) * f], gu[F:][rank * f:(rank + 1) * f]], 0).contiguous()
            t[p + "ffn.down.weight"] = full.w(p + "ffn.down.weight")[:, rank * f:(rank + 1) * f].contiguous()
        return cls(t, full.lowp.dtype)

    @classmethod
    def layered(cls, cfg, device, dtype=None, tensors: dict | None = None, seed: int = 0) -> "InferenceWeights":
        """Weights of a layered decoder (models.layered.LayeredConfig) in the layout of the serving kernels: one packed
        projection for everything that reads the same input (`packed_columns`), experts stacked as [E, 2 ff, d] (gate over up)
        and [E, d, ff], the head padded to whole GEMM tiles; per-channel and per-head constants of recurrent layers in fp32.
        `tensors`: an unsharded checkpoint under `cfg.tensor_shapes()` names, loaded strictly; None: random initialisation on
        the device.  `dtype`: bf16 or fp32 (default: bf16 on a GPU).  Layers that share another's tensors have none here."""
        from ..core.errors import SerializationError, ShapeMismatch
        dev = torch.device(device)
        dt = dtype or (torch.bfloat16 if dev.type == "cuda" else torch.float32)
        shapes = cfg.tensor_shapes()
        if tensors is not None:
            missing = [k for k in shapes if k not in tensors]
            extra = [k for k in tensors if k not in shapes and k not in cfg.unused_tensors()]
            if missing:
                raise SerializationError(f"missing keys: {missing}")
            if extra:
                raise SerializationError(f"unexpected keys: {extra}")
            for k, want in shapes.items():
                if tuple(tensors[k].shape) != tuple(want) and tensors[k].numel() != math.prod(want):
                    raise ShapeMismatch(want, tensors[k].shape, k)

        def get(name, dt=dt):
            shape = shapes[name]
            if tensors is not None:
                return tensors[name].reshape(shape).to(dev, dt)
            last = name.rsplit(".", 1)[-1]
            if last == "correction" or (cfg.design.norm == "rms" and (last in ("norm1", "norm1b", "norm2", "norm2b") or name == "final.norm")):
                return torch.zeros(shape, dtype=dt, device=dev)
            if last in ("norm", "norm1", "norm2", "out", "D"):
                return torch.ones(shape, dtype=dt, device=dev)
            if last in ("r1", "r2"):
                return torch.full(shape, 0.5, dtype=dt, device=dev)
            if last == "b" and len(shape) == 1 and not name.endswith(".dt.b"):
                return torch.zeros(shape, dtype=dt, device=dev)
            if last in ("vmix", "alpha"):
                return torch.full(shape, 0.5, dtype=dt, device=dev)
            g = torch.Generator(device=dev).manual_seed(zlib.crc32(f"{seed}/{name}".encode()))
            if last == "A_log":
                return torch.empty(shape, dtype=torch.float32, device=dev).uniform_(1.0, 16.0, generator=g).log().to(dt)
            if last == "dt_bias" or name.endswith(".dt.b"):
                return torch.empty(shape, dtype=torch.float32, device=dev).uniform_(-6.0, -2.0, generator=g).to(dt)
            std = shape[-1] ** -0.5 if last == "conv" else cfg.init_std
            return torch.empty(shape, dtype=torch.float32, device=dev).normal_(0.0, std, generator=g).to(dt)

        def f32(name):
            return get(name, torch.float32).contiguous()

        def gate_up(p, ff, out):
            """gate rows over up rows; a hidden size that is not a multiple of 8 gets zero rows (act(0) * 0 = 0)."""
            f8 = out.shape[0] // 2
            out[:ff] = get(p + "gate")
            out[f8:f8 + ff] = get(p + "up")

        d = cfg.d_model
        t = {"head": torch.zeros((cfg.vocab_padded, d), dtype=dt, device=dev)}
        if cfg.design.tied:
            t["head"][:cfg.vocab_size] = get("embed")
            t["embed"] = t["head"][:cfg.vocab_size]
        else:
            t["embed"] = get("embed")
            t["head"][:cfg.vocab_size] = get("head")

        def norm(name):
            if cfg.design.norm == "rms":
                t[name] = 1.0 + f32(name)                  # stored as the difference from one
            elif cfg.design.norm == "gain":
                t[name] = f32(name).expand(d).contiguous()
            elif cfg.design.norm == "dyt":
                t[name], t[name + ".b"], t[name + ".alpha"] = f32(name), f32(name + ".b"), f32(name + ".alpha").reshape(1)
            else:
                t[name], t[name + ".b"] = get(name), get(name + ".b")

        def experts(p, m):
            """Router and stacked experts of one layer."""
            t[p + "moe.router"] = get(p + "mlp.router")
            if m.correction:
                t[p + "moe.correction"] = f32(p + "mlp.correction")
            f8 = up8(m.ff)
            w1 = torch.zeros((m.experts, 2 * f8, d), dtype=dt, device=dev)
            w2 = torch.zeros((m.experts, d, f8), dtype=dt, device=dev)
            for e in range(m.experts):
                gate_up(f"{p}mlp.e{e}.", m.ff, w1[e])
                w2[e, :, :m.ff] = get(f"{p}mlp.e{e}.down")
            t[p + "moe.w1"], t[p + "moe.w2"] = w1, w2

        norm("final.norm")
        if cfg.loop is not None:
            t["loop.in"], t["loop.step"] = get("loop.in"), get("loop.step")
        for i, s in enumerate(cfg.layers):
            if cfg.owner(i) != i:
                continue
            if cfg.design.block == "parallel":
                norm(f"l{i}.norm1")
                cls._parallel_block(t, f"l{i}.", s, d, get, f32, dt, dev)
                continue
            p, m = f"l{i}.", s.mlp
            norm(p + "norm1")
            if cfg.design.block in ("sandwich", "pre"):
                sandwich = cfg.design.block == "sandwich"
                if sandwich:
                    norm(p + "norm1b")
                (cls._mixer_in_front if sandwich else cls._mixer_pre)(t, p, s.mixer, d, get, f32, dt, dev)
                if m is not None:
                    norm(p + "norm2")
                    if sandwich:
                        norm(p + "norm2b")
                    if isinstance(m, DenseSpec):
                        t[p + "up"], t[p + "down"] = _pitched(get(p + "mlp.up")), _pitched(get(p + "mlp.down"))
                    else:
                        experts(p, m)
                continue
            t[p + "attn.in"] = torch.cat([get(p + "mix." + c) for c in "qkvg"], 0)
            t[p + "attn.out"] = get(p + "mix.o")
            t[p + "attn.q_norm"], t[p + "attn.k_norm"] = get(p + "mix.q.norm"), get(p + "mix.k.norm")
            if s.mixer.v_mix:
                t[p + "attn.mix"] = get(p + "mix.vmix").float().reshape(1).contiguous()
            if m is None:
                continue
            norm(p + "norm2")
            experts(p, m)
            if m.shared_ff:
                f8 = up8(m.shared_ff)
                w1 = torch.zeros((2 * f8, d), dtype=dt, device=dev)
                gate_up(p + "mlp.shared.", m.shared_ff, w1)
                w2 = torch.zeros((d, f8), dtype=dt, device=dev)
                w2[:, :m.shared_ff] = get(p + "mlp.shared.down")
                t[p + "shared.in"], t[p + "shared.out"] = w1, w2
        return cls(t, dt)

    @staticmethod
    def _mixer_in_front(t, p, m, d, get, f32, dt, dev) -> None:
        """The mixer of a layer with a norm in front: one packed projection of everything that reads it (`latent_columns` for
        latent attention, whose key and value products of all heads are stacked)."""
        x = p + "mix."
        t[p + "attn.out"] = _pitched(get(x + "o"))
        if not isinstance(m, LatentSpec):
            t[p + "attn.in"] = torch.cat([get(x + c) for c in "qkv"], 0)
            if m.bias:
                t[p + "attn.in.b"] = torch.cat([get(x + c + ".b") for c in "qkv"], 0)
            return
        cols = latent_columns(m)
        w = torch.zeros((cols["end"][0], d), dtype=dt, device=dev)
        for nm, src in (("q", "dq"), ("kv", "dkv"), ("g", "g")):
            if nm in cols:
                w[cols[nm][0]:cols[nm][0] + cols[nm][1]] = get(x + src)
        t[p + "attn.in"] = w
        t[p + "attn.q_norm"], t[p + "attn.kv_norm"] = f32(x + "dq.norm"), f32(x + "dkv.norm")
        t[p + "attn.uq"] = _pitched(get(x + "uq"))
        t[p + "attn.ukv"] = _pitched(torch.cat([get(x + "uk"), get(x + "uv")], 0))

    @staticmethod
    def _mixer_pre(t, p, m, d, get, f32, dt, dev) -> None:
        """The mixer of a layer whose output is added as it is: one packed projection of everything that reads the norm (`mixer_columns`),
        and one output projection (both sides of a parallel mixer as one product over their joined outputs)."""
        x = p + "mix."
        if isinstance(m, AttentionSpec):
            own = "qkv" if m.kv_from is None else "q"
            t[p + "attn.in"] = torch.cat([get(x + c) for c in own], 0)
            t[p + "attn.out"] = _pitched(get(x + "o"))
            if m.bias:
                t[p + "attn.in.b"] = torch.cat([get(x + c + ".b") for c in own], 0)
            if m.out_bias:
                t[p + "attn.out.b"] = get(x + "o.b")
            if m.conv:
                t[p + "attn.conv"] = torch.cat([f32(x + c + ".conv") for c in own], 0)
            t.update({f"{p}attn.{c}_norm": f32(f"{x}{c}.norm") for c in own if c != "v"})
            t[p + "attn.r1"], t[p + "attn.r2"] = f32(x + "r1"), f32(x + "r2")
            return
        cols = mixer_columns(m)
        w = torch.zeros((cols["end"][0], d), dtype=dt, device=dev)
        if isinstance(m, RetentionSpec):
            parts = {c: get(x + c) for c in "qkvg"}
            t[p + "attn.out"] = _pitched(get(x + "o"))
            t[p + "attn.decay"] = torch.tensor(m.decay, dtype=torch.float32, device=dev)
        else:
            r, s = x + "right.", m.right
            both = get(r + "in")
            parts = {"q": get(x + "left.q"), "k": get(x + "left.k"), "conv": both[:s.inner], "z": both[s.inner:]}
            t[p + "attn.q_norm"], t[p + "attn.k_norm"] = get(x + "left.q.norm"), get(x + "left.k.norm")
            n = m.left.heads * m.left.vdim
            out = torch.zeros((d, up8(n) + up8(s.inner)), dtype=dt, device=dev)
            out[:, :n], out[:, up8(n):up8(n) + s.inner] = get(x + "left.o"), get(r + "o")
            t[p + "attn.out"] = out
            r8 = up8(s.dt_rank)                            # the rows behind the step sizes' are zero, and so is what they give
            low = torch.zeros((up8(r8 + 2 * s.state), s.inner), dtype=dt, device=dev)
            src = get(r + "x")
            low[:s.dt_rank], low[r8:r8 + 2 * s.state] = src[:s.dt_rank], src[s.dt_rank:]
            t[p + "scan.x"] = _pitched(low)
            step = torch.zeros((s.inner, r8), dtype=dt, device=dev)
            step[:, :s.dt_rank] = get(r + "dt")
            t[p + "scan.dt"] = step
            t[p + "scan.conv"], t[p + "scan.conv.b"] = f32(r + "conv"), f32(r + "conv.b")
            t[p + "scan.dt.b"], t[p + "scan.D"] = f32(r + "dt.b"), f32(r + "D")
            t[p + "scan.A"] = -torch.exp(f32(r + "A_log"))
        for nm, part in parts.items():
            w[cols[nm][0]:cols[nm][0] + cols[nm][1]] = part
        t[p + "attn.in"] = w

    @staticmethod
    def _parallel_block(t, p, s, d, get, f32, dt, dev) -> None:
        """One layer whose mixer and feed-forward read the same input (`packed_columns` gives the columns)."""
        cols, gates = packed_columns(s)
        x = p + "mix."
        par = isinstance(s.mixer, ParallelSpec)
        parts = {"gate": p + "mlp.gate", "up": p + "mlp.up"}
        if par:
            w_in = get(x + "right.in")
            inner, ch = s.mixer.right.inner, s.mixer.right.channels
            parts.update({"q": x + "left.q", "k": x + "left.k", "v": x + "left.v", "z": w_in[:inner], "conv": w_in[inner:inner + ch]})
            small = {"g": x + "left.g", "dt": w_in[inner + ch:]}
        else:
            parts.update({"q": x + "q", "k": x + "k", "v": x + "v", "z": x + "g"})
            small = {"b": x + "b", "a": x + "a"}
        for name, table, src in (("in", cols, parts), ("gates", gates, small)):
            w = torch.zeros((table["end"][0], d), dtype=dt, device=dev)
            for nm, (lo, n) in table.items():
                if nm != "end":
                    part = src[nm]
                    w[lo:lo + n] = get(part) if isinstance(part, str) else part
            t[p + name] = w
        if par:
            r = x + "right."
            t[p + "left.o"], t[p + "right.o"] = get(x + "left.o"), get(r + "o")
            t[p + "left.out"], t[p + "right.out"] = f32(x + "left.out"), f32(x + "right.out")
            t[p + "conv"], t[p + "conv.b"] = f32(r + "conv"), f32(r + "conv.b")
            for nm in ("dt_bias", "A_log", "D", "norm"):
                t[p + nm] = f32(r + nm)
            if s.mlp is not None:
                t[p + "down"] = torch.zeros((d, up8(s.mlp.ff)), dtype=dt, device=dev)
                t[p + "down"][:, :s.mlp.ff] = get(p + "mlp.down")
            return
        t[p + "conv"] = torch.cat([f32(x + c + ".conv") for c in "qkv"], 0)
        for nm in ("dt_bias", "A_log", "norm"):
            t[p + nm] = f32(x + nm)
        # mixer and feed-forward outputs are added anyway: one product over the joined columns
        n = s.mixer.heads * s.mixer.vdim
        t[p + "out"] = torch.zeros((d, up8(n) + (up8(s.mlp.ff) if s.mlp is not None else 0)), dtype=dt, device=dev)
        t[p + "out"][:, :n] = get(x + "o")
        if s.mlp is not None:
            t[p + "out"][:, up8(n):up8(n) + s.mlp.ff] = get(p + "mlp.down")


def packed_columns(s) -> tuple:
    """Columns of the two products over a parallel block's input: ({name: (first, count)} of the one in the activation dtype,
    the same for the one whose results stay fp32: step sizes, decays and per-head gates).  "end": (total, 0).  Sections start at
    multiples of 8; what the convolution reads is contiguous ("conv"; for a delta mixer that is q, k and v)."""
    m = s.mixer
    if isinstance(m, ParallelSpec):
        a, r = m.left, m.right
        groups = [[("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)], [("z", r.inner)], [("conv", r.channels)]]
        small = [[("g", a.heads)], [("dt", r.heads)]]
    else:
        groups = [[("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.heads * m.vdim)], [("z", m.heads * m.vdim)]]
        small = [[("b", m.heads)], [("a", m.heads)]]
    if s.mlp is not None:
        groups.append([("gate", s.mlp.ff)])
        groups.append([("up", s.mlp.ff)])

    def place(groups):
        out, at = {}, 0
        for g in groups:
            for nm, n in g:
                out[nm] = (at, n)
                at += n
            at = up8(at)
        out["end"] = (at, 0)
        return out
    return place(groups), place(small)


def latent_columns(m) -> dict:
    """Columns of the packed projection of a latent attention layer: query latent, cached vector with the shared key part, gate; every
    section starts at a multiple of 8."""
    out, at = {}, 0
    for nm, n in (("q", m.q_rank), ("kv", m.cached), ("g", m.heads * m.vdim if m.gate == "element" else 0)):
        if n:
            out[nm] = (at, n)
            at = up8(at + n)
    out["end"] = (at, 0)
    return out


def mixer_columns(m) -> dict:
    """Columns of the packed projection of a retention or parallel mixer (sections start at multiples of 8).  Retention: what the state
    takes up and reads is contiguous (v, k, q).  Parallel: "v", behind "end", is no product but the room for a copy of the keys."""
    if isinstance(m, RetentionSpec):
        groups = [[("v", m.heads * m.vdim), ("k", m.heads * m.dim), ("q", m.heads * m.dim)], [("g", m.heads * m.vdim)]]
    else:
        a, r = m.left, m.right
        groups = [[("q", a.heads * a.dim), ("k", a.kv_heads * a.dim)], [("conv", r.inner)], [("z", r.inner)]]
    out, at = {}, 0
    for g in groups:
        for nm, n in g:
            out[nm] = (at, n)
            at += n
        at = up8(at)
    out["end"] = (at, 0)
    if not isinstance(m, RetentionSpec):
        out["v"] = (at, m.left.kv_heads * m.left.vdim)
    return out


def _pitched(w: torch.Tensor) -> torch.Tensor:
    """The same matrix with rows that start at multiples of 8 elements (a view of a wider buffer where its own are not)."""
    if w.shape[1] % 8 == 0:
        return w
    out = torch.zeros((w.shape[0], up8(w.shape[1])), dtype=w.dtype, device=w.device)
    out[:, :w.shape[1]] = w
    return out[:, :w.shape[1]]
