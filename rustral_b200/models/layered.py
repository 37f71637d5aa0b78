"""Configuration of layered decoders: models whose config lists every layer with its own mixer and feed-forward sizes.

The first design of this kind is Dolurax: chunked attention with capped scores, a linear distance bias, query / key norms,
values mixed with those of the first mixing layer and an output gate; routed experts with group-limited choice and a shared
expert; a LayerNorm on every sublayer's output, added to a 32-bit residual; scaled and capped logits.  Everything that a
`config.json` can set is a field here; the mechanisms themselves live with their kernels and take these as parameters.
"""
from __future__ import annotations

from dataclasses import asdict, dataclass


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int                     # query / key size of a head
    vdim: int                    # value size of a head
    scale: float
    softcap: float = 0.0         # 0: scores are not capped
    chunk: int = 0               # 0: every earlier position is visible
    v_mix: bool = False          # values are mixed with those of the first layer that has this set

    def __post_init__(self):
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads or self.chunk < 0:
            raise ValueError(f"invalid attention layer: {self}")

    @property
    def packed(self) -> int:
        """Columns of the packed projection [q | k | v | gate]."""
        return self.heads * (self.dim + self.vdim) + self.kv_heads * (self.dim + self.vdim)


@dataclass(frozen=True)
class MoESpec:
    ff: int                      # hidden size of an expert
    experts: int
    top: int
    groups: int = 1              # equal groups of neighbouring experts ...
    keep: int = 1                # ... of which the best `keep` can be chosen from
    shared_ff: int = 0           # hidden size of the expert that every token uses (0: none)

    def __post_init__(self):
        if self.experts % self.groups or not 1 <= self.keep <= self.groups or \
                not 1 <= self.top <= self.keep * (self.experts // self.groups):
            raise ValueError(f"invalid routed feed-forward: {self}")


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec
    mlp: MoESpec | None = None


@dataclass(frozen=True)
class LayeredConfig:
    vocab_size: int
    d_model: int
    layers: tuple
    norm_eps: float = 1e-5
    logit_scale: float = 1.0
    logit_softcap: float = 0.0   # 0: logits are not capped
    seq_len: int = 131072        # longest sequence the engine admits (the design itself has no limit)
    init_std: float = 0.02
    vocab_multiple: int = 128    # rows of the output head are padded to this multiple for aligned GEMM tiles
    arch: str = "Dolurax"

    def __post_init__(self):
        if not self.layers or self.vocab_size < 1 or self.d_model < 8 or self.d_model % 8:
            raise ValueError("layered decoder: at least one layer, and a width that is a multiple of 8")
        if len({s.mixer.kv_heads * s.mixer.vdim for s in self.layers if s.mixer.v_mix}) > 1:
            raise ValueError("layers that mix values must have the same number of value columns")

    @property
    def n_layer(self) -> int:
        return len(self.layers)

    @property
    def vocab_padded(self) -> int:
        m = self.vocab_multiple
        return (self.vocab_size + m - 1) // m * m

    @property
    def first_mix(self) -> int:
        """Index of the first layer that mixes values (its own are the ones the others mix in), -1 without any."""
        return next((i for i, s in enumerate(self.layers) if s.mixer.v_mix), -1)

    def num_parameters(self) -> int:
        n = 2 * self.vocab_size * self.d_model + 2 * self.d_model
        for s in self.layers:
            a, m = s.mixer, s.mlp
            n += a.packed * self.d_model + a.heads * a.vdim * self.d_model + 2 * a.dim + 2 * self.d_model
            if m is not None:
                n += 3 * self.d_model * (m.experts * m.ff + m.shared_ff) + m.experts * self.d_model + 2 * self.d_model
        return n

    def to_dict(self) -> dict:
        return asdict(self)

    # ---- config.json --------------------------------------------------------------------------------------------
    @classmethod
    def from_json(cls, d: dict, **overrides) -> "LayeredConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            if e.get("type", "attention") != "attention":
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            m = e["mixer"]
            mixer = AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                  scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0),
                                  chunk=int((m.get("mask") or {}).get("size") or 0), v_mix=bool(m.get("v_mix", False)))
            mlp = None
            f = e.get("mlp")
            if f is not None:
                if f.get("kind", "moe") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
                r, g = f["router"], f["router"].get("groups") or {}
                mlp = MoESpec(ff=int(f["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]),
                              groups=int(g.get("count", 1)), keep=int(g.get("keep", 1)),
                              shared_ff=int((f.get("shared") or {}).get("ff") or 0))
            layers.append(LayerSpec(mixer, mlp))
        kw = dict(vocab_size=int(d["vocab"]), d_model=int(d["width"]), layers=tuple(layers), norm_eps=float(d["norm"]["eps"]),
                  logit_scale=float(d.get("logit_scale", 1.0)), logit_softcap=float(d.get("logit_softcap") or 0.0),
                  arch=d.get("architecture", "Dolurax"))
        kw.update(overrides)
        return cls(**kw)

    def to_json(self) -> dict:
        """The `config.json` form (inverse of `from_json`)."""
        def layer(s):
            a, m = s.mixer, s.mlp
            mixer = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale, "v_mix": a.v_mix}
            if a.softcap:
                mixer["softcap"] = a.softcap
            if a.chunk:
                mixer["mask"] = {"size": a.chunk}
            mlp = None
            if m is not None:
                router = {"experts": m.experts, "top": m.top}
                if m.groups > 1:
                    router["groups"] = {"count": m.groups, "keep": m.keep}
                mlp = {"kind": "moe", "expert": {"ff": m.ff}, "router": router}
                if m.shared_ff:
                    mlp["shared"] = {"ff": m.shared_ff}
            return {"type": "attention", "mixer": mixer, "mlp": mlp}
        return {"architecture": self.arch, "vocab": self.vocab_size, "width": self.d_model, "norm": {"eps": self.norm_eps},
                "logit_scale": self.logit_scale, "logit_softcap": self.logit_softcap or None,
                "layers": [layer(s) for s in self.layers]}

    # ---- checkpoint tensors ---------------------------------------------------------------------------------------
    def tensor_shapes(self) -> dict:
        """Checkpoint tensor name -> shape (linear weights are [out, in])."""
        d = self.d_model
        t = {"embed": (self.vocab_size, d)}

        def norm(name):
            t[name] = (d,)
            t[name + ".b"] = (d,)

        def ffn(p, ff):
            t[p + "gate"], t[p + "up"], t[p + "down"] = (ff, d), (ff, d), (d, ff)

        for i, s in enumerate(self.layers):
            p, a, m = f"l{i}.", s.mixer, s.mlp
            norm(p + "norm1")
            for nm, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim), ("g", a.heads * a.vdim)):
                t[p + "mix." + nm] = (rows, d)
            t[p + "mix.o"] = (d, a.heads * a.vdim)
            t[p + "mix.q.norm"] = t[p + "mix.k.norm"] = (a.dim,)
            if a.v_mix:
                t[p + "mix.vmix"] = ()
            if m is not None:
                norm(p + "norm2")
                t[p + "mlp.router"] = (m.experts, d)
                for e in range(m.experts):
                    ffn(f"{p}mlp.e{e}.", m.ff)
                if m.shared_ff:
                    ffn(p + "mlp.shared.", m.shared_ff)
        norm("final.norm")
        t["head"] = (self.vocab_size, d)
        return t

    def unused_tensors(self) -> set:
        """Names a checkpoint may hold although no layer reads them: the mixing share of a layer that does not mix, the
        second norm of a layer without a feed-forward."""
        out = set()
        for i, s in enumerate(self.layers):
            if not s.mixer.v_mix:
                out.add(f"l{i}.mix.vmix")
            if s.mlp is None:
                out |= {f"l{i}.norm2", f"l{i}.norm2.b"}
        return out


def uniform_layers(n: int, mixer: dict, mlp: dict | None) -> tuple:
    """`n` equal layers (presets)."""
    return tuple(LayerSpec(AttentionSpec(**mixer), MoESpec(**mlp) if mlp else None) for _ in range(n))
