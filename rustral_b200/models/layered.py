"""Configuration of layered decoders: models whose config lists every layer with its own mixer and feed-forward sizes.

Everything that a `config.json` can set is a field here; what a design fixes is in `DESIGNS`; the mechanisms themselves live
with their kernels and take these as parameters.

Dolurax: chunked attention with capped scores, a linear distance bias, query / key norms, values mixed with those of the first
mixing layer and an element-wise output gate; routed experts with group-limited choice and a shared expert; a LayerNorm on
every sublayer's output, added to a 32-bit residual; scaled and capped logits.

Vafodra: one element-wise "norm" (dynamic tanh) in front of a layer whose mixer and dense feed-forward both read its output and
are added to the residual together; mixers are sliding-window attention (first tokens kept, a sink in the softmax, one output
gate per head) side by side with a Mamba-2 state-space mixer, or a gated delta rule; layers can share another one's tensors.
"""
from __future__ import annotations

from dataclasses import asdict, dataclass


def up8(n: int) -> int:
    return (n + 7) // 8 * 8


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
    window: int = 0              # > 0: a position sees the last `window` positions (itself included) ...
    keep_first: int = 0          # ... and the first `keep_first` of the sequence
    qk_norm: bool = True         # RMS norm of every query and key head
    distance_bias: bool = True   # a linear distance bias with one slope per head
    sink: bool = False           # a further score 0 without a value in the softmax
    gate: str = "element"        # sigmoid output gate: one number per value column ("element") or per head ("head")

    def __post_init__(self):
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads or self.chunk < 0:
            raise ValueError(f"invalid attention layer: {self}")
        if self.window < 0 or self.keep_first < 0 or (self.window and self.chunk) or self.gate not in ("element", "head"):
            raise ValueError(f"invalid attention layer: {self}")

    @property
    def packed(self) -> int:
        """Columns of the packed projection: q, k, v and an element-wise gate."""
        return self.heads * self.dim + self.kv_heads * (self.dim + self.vdim) + (self.heads * self.vdim if self.gate == "element" else 0)

    def tensor_shapes(self, p: str, d: int) -> dict:
        gate = self.heads * self.vdim if self.gate == "element" else self.heads
        t = {p + "q": (self.heads * self.dim, d), p + "k": (self.kv_heads * self.dim, d), p + "v": (self.kv_heads * self.vdim, d),
             p + "g": (gate, d), p + "o": (d, self.heads * self.vdim)}
        if self.qk_norm:
            t[p + "q.norm"] = t[p + "k.norm"] = (self.dim,)
        if self.v_mix:
            t[p + "vmix"] = ()
        return t

    @classmethod
    def from_json(cls, m: dict, **fixed) -> "AttentionSpec":
        mask = m.get("mask") or {}
        size = int(mask.get("size") or 0)
        sliding = fixed.pop("sliding", False)
        return cls(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                   softcap=float(m.get("softcap") or 0.0), v_mix=bool(m.get("v_mix", False)), chunk=0 if sliding else size,
                   window=size if sliding else 0, keep_first=int(mask.get("keep_first") or 0) if sliding else 0, **fixed)

    def to_json(self) -> dict:
        m = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.v_mix:
            m["v_mix"] = True
        if self.softcap:
            m["softcap"] = self.softcap
        if self.chunk:
            m["mask"] = {"size": self.chunk}
        elif self.window:
            m["mask"] = {"size": self.window, "keep_first": self.keep_first}
        return m


@dataclass(frozen=True)
class StateSpaceSpec:
    """Mamba-2: per head a state [state, vdim] that decays by a data-dependent step and takes up B x^T."""
    heads: int
    vdim: int
    state: int
    groups: int = 1              # heads of a group share B and C
    norm_groups: int = 1         # parts of the gated output norm
    conv: int = 4                # taps of the causal convolution over x, B and C

    def __post_init__(self):
        if min(self.heads, self.vdim, self.state, self.groups, self.norm_groups, self.conv) < 1 or self.heads % self.groups or \
                (self.heads * self.vdim) % self.norm_groups:
            raise ValueError(f"invalid state-space layer: {self}")

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    def tensor_shapes(self, p: str, d: int) -> dict:
        return {p + "in": (self.inner + self.channels + self.heads, d), p + "conv": (self.channels, self.conv),
                p + "conv.b": (self.channels,), p + "dt_bias": (self.heads,), p + "A_log": (self.heads,), p + "D": (self.heads,),
                p + "norm": (self.inner,), p + "o": (d, self.inner)}

    @classmethod
    def from_json(cls, m: dict) -> "StateSpaceSpec":
        return cls(heads=int(m["heads"]), vdim=int(m["vdim"]), state=int(m["state"]), groups=int(m.get("groups", 1)),
                   norm_groups=int(m.get("norm_groups", 1)), conv=int(m["conv"]))

    def to_json(self) -> dict:
        return asdict(self)


@dataclass(frozen=True)
class ParallelSpec:
    """Attention and a state-space mixer side by side: half the sum of their outputs, each RMS-normed over the width."""
    left: AttentionSpec
    right: StateSpaceSpec

    def tensor_shapes(self, p: str, d: int) -> dict:
        return {**self.left.tensor_shapes(p + "left.", d), **self.right.tensor_shapes(p + "right.", d),
                p + "left.out": (d,), p + "right.out": (d,)}

    def to_json(self) -> dict:
        return {"left": self.left.to_json(), "right": self.right.to_json()}


@dataclass(frozen=True)
class DeltaSpec:
    """Gated delta rule: per head a state [dim, vdim] that is decayed and corrected towards v at k."""
    heads: int
    kv_heads: int                # query / key heads; heads / kv_heads value heads share one
    dim: int
    vdim: int
    conv: int = 4

    def __post_init__(self):
        if min(self.heads, self.kv_heads, self.dim, self.vdim, self.conv) < 1 or self.heads % self.kv_heads:
            raise ValueError(f"invalid delta layer: {self}")

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    def tensor_shapes(self, p: str, d: int) -> dict:
        t = {}
        for nm, n in (("q", self.kv_heads * self.dim), ("k", self.kv_heads * self.dim), ("v", self.heads * self.vdim)):
            t[p + nm], t[p + nm + ".conv"] = (n, d), (n, self.conv)
        t.update({p + "b": (self.heads, d), p + "a": (self.heads, d), p + "A_log": (self.heads,), p + "dt_bias": (self.heads,),
                  p + "norm": (self.vdim,), p + "g": (self.heads * self.vdim, d), p + "o": (d, self.heads * self.vdim)})
        return t

    @classmethod
    def from_json(cls, m: dict) -> "DeltaSpec":
        return cls(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), conv=int(m["conv"]))

    def to_json(self) -> dict:
        return asdict(self)


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

    def tensor_shapes(self, p: str, d: int) -> dict:
        t = {p + "router": (self.experts, d)}
        for e in range(self.experts):
            t.update(_ffn_shapes(f"{p}e{e}.", self.ff, d))
        if self.shared_ff:
            t.update(_ffn_shapes(p + "shared.", self.shared_ff, d))
        return t

    @classmethod
    def from_json(cls, f: dict) -> "MoESpec":
        r, g = f["router"], f["router"].get("groups") or {}
        return cls(ff=int(f["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]), groups=int(g.get("count", 1)),
                   keep=int(g.get("keep", 1)), shared_ff=int((f.get("shared") or {}).get("ff") or 0))

    def to_json(self) -> dict:
        router = {"experts": self.experts, "top": self.top}
        if self.groups > 1:
            router["groups"] = {"count": self.groups, "keep": self.keep}
        mlp = {"kind": "moe", "expert": {"ff": self.ff}, "router": router}
        if self.shared_ff:
            mlp["shared"] = {"ff": self.shared_ff}
        return mlp


@dataclass(frozen=True)
class DenseSpec:
    ff: int
    act: str = "relu"            # of the gate: act(gate) * up

    def __post_init__(self):
        if self.ff < 1 or self.act not in ("relu", "silu"):
            raise ValueError(f"invalid dense feed-forward: {self}")

    def tensor_shapes(self, p: str, d: int) -> dict:
        return _ffn_shapes(p, self.ff, d)

    def to_json(self) -> dict:
        return {"kind": "dense", "ff": self.ff}


def _ffn_shapes(p: str, ff: int, d: int) -> dict:
    return {p + "gate": (ff, d), p + "up": (ff, d), p + "down": (d, ff)}


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec | ParallelSpec | DeltaSpec
    mlp: MoESpec | DenseSpec | None = None
    weights_of: int | None = None        # the layer whose tensors this one uses (with a cache or state of its own)


@dataclass(frozen=True)
class Design:
    """What a layered design fixes for all its models."""
    mixers: tuple                        # mixer types a layer can have
    mlps: tuple                          # kinds of feed-forward
    block: str                           # "output_norm": norm on every sublayer's output; "parallel": one norm in front of both
    norm: str                            # "layer" or "dyt"
    attention: dict                      # fixed fields of AttentionSpec ("sliding": the mask is a window)
    act: str = "silu"


DESIGNS = {
    "Dolurax": Design(("attention",), ("moe",), "output_norm", "layer", {}),
    "Vafodra": Design(("parallel", "delta"), ("dense",), "parallel", "dyt",
                      dict(sliding=True, qk_norm=False, distance_bias=False, sink=True, gate="head"), act="relu"),
}


@dataclass(frozen=True)
class LayeredConfig:
    vocab_size: int
    d_model: int
    layers: tuple
    norm_eps: float = 1e-5
    logit_scale: float = 1.0
    logit_softcap: float = 0.0   # 0: logits are not capped
    embed_scale: float = 1.0
    residual_mult: float = 1.0   # of what a layer adds to the residual (parallel blocks)
    seq_len: int = 131072        # longest sequence the engine admits (the design itself has no limit)
    init_std: float = 0.02
    vocab_multiple: int = 128    # rows of the output head are padded to this multiple for aligned GEMM tiles
    arch: str = "Dolurax"

    def __post_init__(self):
        if self.arch not in DESIGNS:
            raise ValueError(f"layered decoder: unknown design {self.arch!r}")
        if not self.layers or self.vocab_size < 1 or self.d_model < 1:
            raise ValueError("layered decoder: at least one layer, and a positive width and vocabulary")
        if self.d_model % 8 and any(isinstance(s.mlp, MoESpec) for s in self.layers):
            raise ValueError("layered decoder: the width of a model with routed experts is a multiple of 8")
        mixing = [s.mixer for s in self.layers if getattr(s.mixer, "v_mix", False)]
        if len({a.kv_heads * a.vdim for a in mixing}) > 1:
            raise ValueError("layers that mix values must have the same number of value columns")
        for i, s in enumerate(self.layers):
            o = self.layers[self.owner(i)]
            if (o.mixer, o.mlp) != (s.mixer, s.mlp):
                raise ValueError(f"layer {i} uses the tensors of layer {self.owner(i)}, whose sizes differ")

    @property
    def design(self) -> Design:
        return DESIGNS[self.arch]

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
        return next((i for i, s in enumerate(self.layers) if getattr(s.mixer, "v_mix", False)), -1)

    def owner(self, i: int) -> int:
        """The layer whose tensors layer `i` uses (itself, or where its `weights_of` leads)."""
        for _ in range(len(self.layers)):
            j = self.layers[i].weights_of
            if j is None or j == i:
                return i
            if not 0 <= j < len(self.layers):
                raise ValueError(f"layer {i} refers to layer {j}, which does not exist")
            i = j
        raise ValueError("layers refer to one another's tensors in a circle")

    def num_parameters(self) -> int:
        """Elements of the checkpoint's tensors (shared ones once), without the value mixing shares."""
        n = 0
        for name, shape in self.tensor_shapes().items():
            if not name.endswith("vmix"):
                k = 1
                for s in shape:
                    k *= s
                n += k
        return n

    def to_dict(self) -> dict:
        return asdict(self)

    # ---- config.json --------------------------------------------------------------------------------------------
    @classmethod
    def from_json(cls, d: dict, **overrides) -> "LayeredConfig":
        arch = d.get("architecture", "Dolurax")
        if arch not in DESIGNS:
            raise ValueError(f"layered decoder: unknown design {arch!r}")
        design = DESIGNS[arch]
        layers = []
        for i, e in enumerate(d["layers"]):
            kind, m, f = e.get("type", design.mixers[0]), e["mixer"], e.get("mlp")
            if kind not in design.mixers:
                raise ValueError(f"layer {i}: unknown mixer {kind!r}")
            if kind == "parallel":
                mixer = ParallelSpec(AttentionSpec.from_json(m["left"], **design.attention), StateSpaceSpec.from_json(m["right"]))
            elif kind == "delta":
                mixer = DeltaSpec.from_json(m)
            else:
                mixer = AttentionSpec.from_json(m, **design.attention)
            mlp = None
            if f is not None:
                if f.get("kind", design.mlps[0]) not in design.mlps:
                    raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
                mlp = MoESpec.from_json(f) if design.mlps == ("moe",) else DenseSpec(int(f["ff"]), design.act)
            layers.append(LayerSpec(mixer, mlp, e.get("weights_of")))
        kw = dict(vocab_size=int(d["vocab"]), d_model=int(d["width"]), layers=tuple(layers), norm_eps=float(d["norm"]["eps"]),
                  logit_scale=float(d.get("logit_scale", 1.0)), logit_softcap=float(d.get("logit_softcap") or 0.0),
                  embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                  residual_mult=float(d.get("residual_mult", 1.0)), arch=arch)
        kw.update(overrides)
        return cls(**kw)

    def to_json(self) -> dict:
        """The `config.json` form (inverse of `from_json`)."""
        types = {AttentionSpec: "attention", ParallelSpec: "parallel", DeltaSpec: "delta"}

        def layer(s):
            e = {"type": types[type(s.mixer)], "mixer": s.mixer.to_json(), "mlp": None if s.mlp is None else s.mlp.to_json()}
            if s.weights_of is not None:
                e["weights_of"] = s.weights_of
            return e
        return {"architecture": self.arch, "vocab": self.vocab_size, "width": self.d_model, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embed_scale}, "residual_mult": self.residual_mult,
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
            if self.design.norm == "dyt":
                t[name + ".alpha"] = ()

        for i, s in enumerate(self.layers):
            if self.owner(i) != i:
                continue
            p = f"l{i}."
            norm(p + "norm1")
            t.update(s.mixer.tensor_shapes(p + "mix.", d))
            if s.mlp is not None:
                if self.design.block == "output_norm":
                    norm(p + "norm2")
                t.update(s.mlp.tensor_shapes(p + "mlp.", d))
        norm("final.norm")
        t["head"] = (self.vocab_size, d)
        return t

    def unused_tensors(self) -> set:
        """Names a checkpoint may hold although no layer reads them: the mixing share of a layer that does not mix, the
        second norm of a layer without a feed-forward."""
        out = set()
        if self.design.block != "output_norm":
            return out
        for i, s in enumerate(self.layers):
            if not s.mixer.v_mix:
                out.add(f"l{i}.mix.vmix")
            if s.mlp is None:
                out |= {f"l{i}.norm2", f"l{i}.norm2.b"}
        return out


def uniform_layers(n: int, mixer: dict, mlp: dict | None) -> tuple:
    """`n` equal attention layers with routed experts (presets)."""
    return tuple(LayerSpec(AttentionSpec(**mixer), MoESpec(**mlp) if mlp else None) for _ in range(n))


def hybrid_layers(order: str, left: dict, right: dict, delta: dict, ff: dict, weights_of: dict | None = None) -> tuple:
    """Layers of a Vafodra model: 'p' a parallel mixer (`left`, `right`), 'd' a delta mixer; `ff`: hidden size of the
    feed-forward behind either ({'p': .., 'd': ..}, 0: none); `weights_of`: layer -> owner."""
    fixed = {k: v for k, v in DESIGNS["Vafodra"].attention.items() if k != "sliding"}
    act = DESIGNS["Vafodra"].act
    mixers = {"p": ParallelSpec(AttentionSpec(**left, **fixed), StateSpaceSpec(**right)), "d": DeltaSpec(**delta)}
    return tuple(LayerSpec(mixers[c], DenseSpec(ff[c], act) if ff[c] else None, (weights_of or {}).get(i)) for i, c in enumerate(order))
