"""Configuration of layered decoders: models whose config lists every layer with its own mixer and feed-forward sizes.

Everything that a `config.json` can set is a field here; what a design fixes is in `DESIGNS`; the mechanisms themselves live
with their kernels and take these as parameters.

Dolurax: chunked attention with capped scores, a linear distance bias, query / key norms, values mixed with those of the first
mixing layer and an element-wise output gate; routed experts with group-limited choice and a shared expert; a LayerNorm on
every sublayer's output, added to a 32-bit residual; scaled and capped logits.

Vafodra: one element-wise "norm" (dynamic tanh) in front of a layer whose mixer and dense feed-forward both read its output and
are added to the residual together; mixers are sliding-window attention (first tokens kept, a sink in the softmax, one output
gate per head) side by side with a Mamba-2 state-space mixer, or a gated delta rule; layers can share another one's tensors.

Bikilix: an RMS norm in front of every sublayer and another on its output; sliding-window attention with projection biases and
partial rotary positions, or latent attention (keys and values come from one small cached vector per token) with rotated and
unrotated key parts and an element-wise output gate; dense squared-ReLU feed-forwards or routed experts with clamped gates, chosen by
corrected sigmoid scores; a run of layers can be passed through several times, each pass starting from a product of the stream
and the embedding; the embedding table is the output head.

Seredra: an RMS norm with a single gain in front of every sublayer, outputs added as they are; attention with short convolutions over
queries, keys and values, norms over whole projections, a query temperature and a logarithmic distance bias (keys and values can be
another layer's), retention (a matrix of state per head that decays at one rate), or attention whose values are its keys beside a selective
scan; dense squared-ReLU feed-forwards or routed experts whose sigmoid scores multiply the experts' inputs.
"""
from __future__ import annotations

import math
from dataclasses import asdict, dataclass, field


def up8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass(frozen=True)
class RotarySpec:
    """Rotary positions on the first `dims` numbers of a head: neighbours are paired, or with `half` numbers i and i + dims / 2.
    `factor` > 1: YaRN scaling, which leaves pairs that turn at least `fast` times within `original` positions alone and slows those
    that turn at most `slow` times."""
    dims: int
    base: float
    factor: float = 1.0
    original: int = 0
    fast: float = 32.0
    slow: float = 1.0
    scaled: bool = False
    half: bool = False

    def __post_init__(self):
        if self.dims < 0 or self.dims % 2 or self.base <= 1.0 or (self.scaled and (self.factor <= 0.0 or self.original <= 0 or self.fast <= 0.0
                                                                                   or self.slow <= 0.0)):
            raise ValueError(f"invalid rotary positions: {self}")

    def frequencies(self) -> list:
        """Angle per position of every pair."""
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        if not self.scaled:
            return f

        def place(turns):                 # where (a fractional index) the pairs turn this often within `original` positions
            return self.dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))
        lo, hi = max(math.floor(place(self.fast)), 0), min(math.ceil(place(self.slow)), self.dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(f))]
        return [fi / self.factor * r + fi * (1.0 - r) for fi, r in zip(f, ramp)]

    @property
    def magnitude(self) -> float:
        """Factor on cosines and sines."""
        return 0.1 * math.log(self.factor) + 1.0 if self.scaled else 1.0

    @classmethod
    def from_json(cls, r: dict | None, half: bool = False) -> "RotarySpec | None":
        if not r:
            return None
        s = r.get("scaling")
        kw = dict(factor=float(s["factor"]), original=int(s["original"]), fast=float(s["fast"]), slow=float(s["slow"]), scaled=True) if s else {}
        return cls(dims=int(r["dims"]), base=float(r["base"]), half=half, **kw)

    def to_json(self) -> dict:
        r = {"dims": self.dims, "base": self.base}
        if self.scaled:
            r["scaling"] = {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}
        return r


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
    gate: str = "element"        # sigmoid output gate: one number per value column ("element"), per head ("head"), or "none"
    rot: RotarySpec | None = None        # rotary positions on queries and keys
    bias: bool = False           # the query, key and value projections have biases
    out_bias: bool = False       # the output projection has a bias
    norm_over: str = "head"      # what a query / key norm spans: every "head" by itself, or "all" of the projection
    conv: int = 0                # taps of a causal convolution on every channel of queries, keys and values (0: none)
    temp_coef: float = 0.0       # queries at position p times 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1)
    temp_every: int = 0          # 0: no such factor
    log_bias: bool = False       # r1 * ln(1 + r2 * distance) is taken off the scores, with two numbers per head
    values_are_keys: bool = False        # values: a copy of the unnormed, unrotated keys
    kv_from: int | None = None   # the layer whose cached keys and values are used instead of own ones

    def __post_init__(self):
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads or self.chunk < 0:
            raise ValueError(f"invalid attention layer: {self}")
        if self.window < 0 or self.keep_first < 0 or (self.window and self.chunk) or self.gate not in ("element", "head", "none"):
            raise ValueError(f"invalid attention layer: {self}")
        if self.rot is not None and self.rot.dims > self.dim:
            raise ValueError(f"more rotated dimensions than a head has: {self}")
        if self.norm_over not in ("head", "all") or self.conv < 0 or self.temp_every < 0 or (self.values_are_keys and self.vdim != self.dim):
            raise ValueError(f"invalid attention layer: {self}")

    @property
    def packed(self) -> int:
        """Columns of the packed projection: q, k, v and an element-wise gate."""
        return self.heads * self.dim + self.kv_heads * (self.dim + self.vdim) + (self.heads * self.vdim if self.gate == "element" else 0)

    def tensor_shapes(self, p: str, d: int) -> dict:
        t = {p + "q": (self.heads * self.dim, d), p + "k": (self.kv_heads * self.dim, d), p + "v": (self.kv_heads * self.vdim, d)}
        if self.values_are_keys:
            del t[p + "v"]
        if self.kv_from is not None:
            t = {p + "q": t[p + "q"]}
        own = [c for c in "qkv" if p + c in t]
        if self.gate != "none":
            t[p + "g"] = (self.heads * self.vdim if self.gate == "element" else self.heads, d)
        t[p + "o"] = (d, self.heads * self.vdim)
        if self.bias:
            t.update({p + c + ".b": t[p + c][:1] for c in own})
        if self.out_bias:
            t[p + "o.b"] = (d,)
        if self.conv:
            t.update({p + c + ".conv": (t[p + c][0], self.conv) for c in own})
        if self.qk_norm:
            t.update({p + c + ".norm": (self.dim,) if self.norm_over == "head" else t[p + c][:1] for c in own if c != "v"})
        if self.log_bias:
            t[p + "r1"] = t[p + "r2"] = (self.heads,)
        if self.v_mix:
            t[p + "vmix"] = ()
        return t

    @classmethod
    def from_json(cls, m: dict, **fixed) -> "AttentionSpec":
        mask = m.get("mask") or {}
        size = int(mask.get("size") or 0)
        sliding, half = fixed.pop("sliding", False), fixed.pop("half", False)
        temp = m.get("q_temp") or {}
        return cls(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                   softcap=float(m.get("softcap") or 0.0), v_mix=bool(m.get("v_mix", False)), chunk=0 if sliding else size,
                   window=size if sliding else 0, keep_first=int(mask.get("keep_first") or 0) if sliding else 0,
                   rot=RotarySpec.from_json(m.get("rot"), half), conv=int(m.get("conv") or 0), temp_coef=float(temp.get("coef", 0.0)),
                   temp_every=int(temp.get("every", 0)), kv_from=None if m.get("kv_from") is None else int(m["kv_from"]), **fixed)

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
        if self.rot is not None:
            m["rot"] = self.rot.to_json()
        if self.conv:
            m["conv"] = self.conv
        if self.temp_every:
            m["q_temp"] = {"coef": self.temp_coef, "every": self.temp_every}
        if self.kv_from is not None:
            m["kv_from"] = self.kv_from
        return m


@dataclass(frozen=True)
class LatentSpec:
    """Latent attention: keys (their unrotated part) and values of all heads are products of one normed vector per token, which is
    what the cache holds beside a rotated key part that the heads share.  Queries come through a normed vector of their own."""
    heads: int
    dim: int                     # unrotated query / key size of a head
    rot_dim: int                 # rotated query / key size
    vdim: int
    kv_rank: int                 # size of the cached vector
    q_rank: int
    scale: float
    rot: RotarySpec
    gate: str = "element"        # sigmoid output gate, one number per value column ("none": no gate)

    def __post_init__(self):
        if min(self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank, self.q_rank) < 1 or self.rot.dims > self.rot_dim or \
                self.gate not in ("element", "none"):
            raise ValueError(f"invalid latent attention layer: {self}")

    @property
    def qk_dim(self) -> int:
        return self.dim + self.rot_dim

    @property
    def cached(self) -> int:
        """Numbers per token in the cache."""
        return self.kv_rank + self.rot_dim

    def tensor_shapes(self, p: str, d: int) -> dict:
        H = self.heads
        t = {p + "dq": (self.q_rank, d), p + "dq.norm": (self.q_rank,), p + "uq": (H * self.qk_dim, self.q_rank),
             p + "dkv": (self.cached, d), p + "dkv.norm": (self.kv_rank,), p + "uk": (H * self.dim, self.kv_rank),
             p + "uv": (H * self.vdim, self.kv_rank), p + "o": (d, H * self.vdim)}
        if self.gate == "element":
            t[p + "g"] = (H * self.vdim, d)
        return t

    @classmethod
    def from_json(cls, m: dict) -> "LatentSpec":
        return cls(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                   q_rank=int(m["q_rank"]), scale=float(m["scale"]), rot=RotarySpec.from_json(m["rot"]))

    def to_json(self) -> dict:
        m = {k: getattr(self, k) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale")}
        return {**m, "rot": self.rot.to_json()}


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
class SelectiveSpec:
    """Mamba: per channel a state of `state` numbers that decay and take up the input with a step size of the channel's own; step sizes
    (through `dt_rank` numbers), B and C come from the channels behind the convolution."""
    inner: int
    state: int
    dt_rank: int
    conv: int = 4                # taps of the causal convolution over the channels

    def __post_init__(self):
        if min(self.inner, self.state, self.dt_rank, self.conv) < 1:
            raise ValueError(f"invalid selective scan: {self}")

    def tensor_shapes(self, p: str, d: int) -> dict:
        return {p + "in": (2 * self.inner, d), p + "conv": (self.inner, self.conv), p + "conv.b": (self.inner,),
                p + "x": (self.dt_rank + 2 * self.state, self.inner), p + "dt": (self.inner, self.dt_rank), p + "dt.b": (self.inner,),
                p + "A_log": (self.inner, self.state), p + "D": (self.inner,), p + "o": (d, self.inner)}

    @classmethod
    def from_json(cls, m: dict) -> "SelectiveSpec":
        return cls(inner=int(m["inner"]), state=int(m["state"]), dt_rank=int(m["dt_rank"]), conv=int(m["conv"]))

    def to_json(self) -> dict:
        return asdict(self)


@dataclass(frozen=True)
class ParallelSpec:
    """Attention and a recurrent mixer side by side: half the sum of their outputs, each RMS-normed over the width, or with `scales` the
    outputs as they are times one number each."""
    left: AttentionSpec
    right: StateSpaceSpec | SelectiveSpec
    scales: tuple | None = None

    def tensor_shapes(self, p: str, d: int) -> dict:
        t = {**self.left.tensor_shapes(p + "left.", d), **self.right.tensor_shapes(p + "right.", d)}
        return t if self.scales is not None else {**t, p + "left.out": (d,), p + "right.out": (d,)}

    def to_json(self) -> dict:
        m = {"left": self.left.to_json(), "right": self.right.to_json()}
        return m if self.scales is None else {**m, "left_scale": self.scales[0], "right_scale": self.scales[1]}


@dataclass(frozen=True)
class RetentionSpec:
    """Retention: every head multiplies its state [dim, vdim] by a constant of its own and takes up k v^T; what a query reads from it is
    normed by itself and gated."""
    heads: int
    dim: int
    vdim: int
    decay: tuple
    rot: RotarySpec | None = None

    def __post_init__(self):
        if min(self.heads, self.dim, self.vdim) < 1 or len(self.decay) != self.heads or not all(0.0 < x <= 1.0 for x in self.decay) or \
                (self.rot is not None and self.rot.dims > self.dim):
            raise ValueError(f"invalid retention layer: {self}")

    def tensor_shapes(self, p: str, d: int) -> dict:
        n, nv = self.heads * self.dim, self.heads * self.vdim
        return {p + "q": (n, d), p + "k": (n, d), p + "v": (nv, d), p + "g": (nv, d), p + "o": (d, nv)}

    @classmethod
    def from_json(cls, m: dict, half: bool = False) -> "RetentionSpec":
        return cls(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), decay=tuple(float(x) for x in m["decay"]),
                   rot=RotarySpec.from_json(m.get("rot"), half))

    def to_json(self) -> dict:
        m = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}
        return m if self.rot is None else {**m, "rot": self.rot.to_json()}


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
    score: str = "softmax"       # router scores: "softmax" over the experts, or "sigmoid" of every logit by itself
    correction: bool = False     # a vector is added to the scores for the choice, not for the weights
    group_best: int = 1          # a group counts as the sum of its this many largest choice scores
    renorm: bool = True          # weights are divided by their sum
    act: str = "silu"            # act(gate) * up; "clamped": see ops.moe.swiglu_rows
    limit: float = 0.0           # of the clamped activation
    weigh: str = "output"        # what an expert's weight multiplies: its "output" or its "input"

    def __post_init__(self):
        if self.weigh not in ("output", "input") or self.score not in ("softmax", "sigmoid") or self.act not in ("silu", "clamped") or self.group_best not in (1, 2) or \
                (self.score == "softmax" and (self.correction or self.group_best != 1)) or (self.act == "clamped") != (self.limit > 0.0):
            raise ValueError(f"invalid routed feed-forward: {self}")
        if self.experts % self.groups or not 1 <= self.keep <= self.groups or \
                not 1 <= self.top <= self.keep * (self.experts // self.groups):
            raise ValueError(f"invalid routed feed-forward: {self}")

    def tensor_shapes(self, p: str, d: int) -> dict:
        t = {p + "router": (self.experts, d)}
        if self.correction:
            t[p + "correction"] = (self.experts,)
        for e in range(self.experts):
            t.update(_ffn_shapes(f"{p}e{e}.", self.ff, d))
        if self.shared_ff:
            t.update(_ffn_shapes(p + "shared.", self.shared_ff, d))
        return t

    @classmethod
    def from_json(cls, f: dict, **fixed) -> "MoESpec":
        r, g = f["router"], f["router"].get("groups") or {}
        return cls(ff=int(f["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]), groups=int(g.get("count", 1)),
                   keep=int(g.get("keep", 1)), shared_ff=int((f.get("shared") or {}).get("ff") or 0),
                   limit=float(f["expert"].get("limit") or 0.0), **fixed)

    def to_json(self) -> dict:
        router = {"experts": self.experts, "top": self.top}
        if self.groups > 1:
            router["groups"] = {"count": self.groups, "keep": self.keep}
        mlp = {"kind": "moe", "expert": {"ff": self.ff}, "router": router}
        if self.limit:
            mlp["expert"]["limit"] = self.limit
        if self.shared_ff:
            mlp["shared"] = {"ff": self.shared_ff}
        return mlp


@dataclass(frozen=True)
class DenseSpec:
    ff: int
    act: str = "relu"            # of the gate: act(gate) * up; not gated: act(up)
    gated: bool = True

    def __post_init__(self):
        if self.ff < 1 or self.act not in (("relu", "silu") if self.gated else ("relu2",)):
            raise ValueError(f"invalid dense feed-forward: {self}")

    def tensor_shapes(self, p: str, d: int) -> dict:
        t = _ffn_shapes(p, self.ff, d)
        return t if self.gated else {k: v for k, v in t.items() if k != p + "gate"}

    def to_json(self) -> dict:
        return {"kind": "dense", "ff": self.ff}


def _ffn_shapes(p: str, ff: int, d: int) -> dict:
    return {p + "gate": (ff, d), p + "up": (ff, d), p + "down": (d, ff)}


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec | ParallelSpec | DeltaSpec | LatentSpec | RetentionSpec
    mlp: MoESpec | DenseSpec | None = None
    weights_of: int | None = None        # the layer whose tensors this one uses (with a cache or state of its own)


@dataclass(frozen=True)
class LoopSpec:
    """Layers start .. stop - 1 run `times` times in a row with the same weights and a cache of their own in each pass."""
    start: int
    stop: int
    times: int

    def __post_init__(self):
        if not 0 <= self.start < self.stop or self.times < 1:
            raise ValueError(f"invalid loop: {self}")


@dataclass(frozen=True)
class Design:
    """What a layered design fixes for all its models."""
    mixers: tuple                        # mixer types a layer can have
    mlps: tuple                          # kinds of feed-forward
    block: str                           # "output_norm": norm on every sublayer's output; "parallel": one norm in front of both;
                                         # "sandwich": a norm in front of every sublayer and one on its output;
                                         # "pre": a norm in front of every sublayer, whose output is added as it is
    norm: str                            # "layer", "dyt", "rms" (weights stored as the difference from one) or "gain" (RMS, one number)
    attention: dict                      # fixed fields of AttentionSpec ("sliding": the mask is a window, "half": of its RotarySpec)
    act: str = "silu"
    experts: dict = field(default_factory=dict)      # fixed fields of MoESpec
    gated: bool = True                   # dense feed-forwards have a gate
    tied: bool = False                   # the embedding table is the output head
    left: dict | None = None             # fixed fields of the attention in a parallel mixer, where they differ
    selective: bool = False              # a parallel mixer's other side is a selective scan, and both sides have scales
    half: bool = False                   # rotary positions of retention pair halves


DESIGNS = {
    "Dolurax": Design(("attention",), ("moe",), "output_norm", "layer", {}),
    "Vafodra": Design(("parallel", "delta"), ("dense",), "parallel", "dyt",
                      dict(sliding=True, qk_norm=False, distance_bias=False, sink=True, gate="head"), act="relu"),
    "Bikilix": Design(("attention", "latent_attention"), ("dense", "moe"), "sandwich", "rms",
                      dict(sliding=True, qk_norm=False, distance_bias=False, gate="none", bias=True), act="relu2",
                      experts=dict(score="sigmoid", correction=True, group_best=2, renorm=False, act="clamped"), gated=False, tied=True),
    "Seredra": Design(("attention", "parallel", "retention"), ("dense", "moe"), "pre", "gain",
                      dict(distance_bias=False, gate="none", bias=True, out_bias=True, norm_over="all", log_bias=True),
                      act="relu2", experts=dict(score="sigmoid", renorm=False, weigh="input"), gated=False,
                      left=dict(distance_bias=False, gate="none", values_are_keys=True, half=True), selective=True, half=True),
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
    loop: LoopSpec | None = None         # layers that run several times

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
            j = getattr(s.mixer, "kv_from", None)
            if j is None:
                continue
            o = self.layers[j].mixer if 0 <= j < i else None
            if not isinstance(o, AttentionSpec) or o.kv_from is not None or (o.kv_heads, o.dim, o.vdim) != (s.mixer.kv_heads, s.mixer.dim, s.mixer.vdim):
                raise ValueError(f"layer {i} cannot use the keys and values of layer {j}")
        if self.loop is not None and (self.loop.stop > len(self.layers) or self.design.block != "sandwich"):
            raise ValueError(f"{self.arch} with {len(self.layers)} layers cannot have {self.loop}")
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
    def runs(self) -> tuple:
        """(layer, number of the pass it opens or None) in the order the layers run."""
        n, lp = self.n_layer, self.loop
        if lp is None:
            return tuple((i, None) for i in range(n))
        body = [(i, t if i == lp.start else None) for t in range(lp.times) for i in range(lp.start, lp.stop)]
        return (*((i, None) for i in range(lp.start)), *body, *((i, None) for i in range(lp.stop, n)))

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
            if kind == "latent_attention":
                mixer = LatentSpec.from_json(m)
            elif kind == "parallel":
                left = AttentionSpec.from_json(m["left"], **(design.attention if design.left is None else design.left))
                if design.selective:
                    mixer = ParallelSpec(left, SelectiveSpec.from_json(m["right"]), (float(m["left_scale"]), float(m["right_scale"])))
                else:
                    mixer = ParallelSpec(left, StateSpaceSpec.from_json(m["right"]))
            elif kind == "retention":
                mixer = RetentionSpec.from_json(m, design.half)
            elif kind == "delta":
                mixer = DeltaSpec.from_json(m)
            else:
                mixer = AttentionSpec.from_json(m, **design.attention)
            mlp = None
            if f is not None:
                fkind = f.get("kind", design.mlps[0])
                if fkind not in design.mlps:
                    raise ValueError(f"layer {i}: unknown feed-forward {fkind!r}")
                mlp = MoESpec.from_json(f, **design.experts) if fkind == "moe" else DenseSpec(int(f["ff"]), design.act, design.gated)
            layers.append(LayerSpec(mixer, mlp, e.get("weights_of")))
        kw = dict(vocab_size=int(d["vocab"]), d_model=int(d["width"]), layers=tuple(layers), norm_eps=float(d["norm"]["eps"]),
                  logit_scale=float(d.get("logit_scale", 1.0)), logit_softcap=float(d.get("logit_softcap") or 0.0),
                  embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                  residual_mult=float(d.get("residual_mult", 1.0)), arch=arch)
        if d.get("loop"):
            kw["loop"] = LoopSpec(**{k: int(d["loop"][k]) for k in ("start", "stop", "times")})
        kw.update(overrides)
        return cls(**kw)

    def to_json(self) -> dict:
        """The `config.json` form (inverse of `from_json`)."""
        types = {AttentionSpec: "attention", ParallelSpec: "parallel", DeltaSpec: "delta", LatentSpec: "latent_attention", RetentionSpec: "retention"}

        def layer(s):
            e = {"type": types[type(s.mixer)], "mixer": s.mixer.to_json(), "mlp": None if s.mlp is None else s.mlp.to_json()}
            if s.weights_of is not None:
                e["weights_of"] = s.weights_of
            return e
        loop = {} if self.loop is None else {"loop": asdict(self.loop)}
        return {"architecture": self.arch, **loop, "vocab": self.vocab_size, "width": self.d_model, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embed_scale}, "residual_mult": self.residual_mult,
                "logit_scale": self.logit_scale, "logit_softcap": self.logit_softcap or None,
                "layers": [layer(s) for s in self.layers]}

    # ---- checkpoint tensors ---------------------------------------------------------------------------------------
    def tensor_shapes(self) -> dict:
        """Checkpoint tensor name -> shape (linear weights are [out, in])."""
        d = self.d_model
        t = {"embed": (self.vocab_size, d)}

        if self.loop is not None:
            t["loop.in"], t["loop.step"] = (d, 2 * d), (self.loop.times, d)

        def norm(name):
            t[name] = () if self.design.norm == "gain" else (d,)
            if self.design.norm not in ("rms", "gain"):
                t[name + ".b"] = (d,)
            if self.design.norm == "dyt":
                t[name + ".alpha"] = ()

        for i, s in enumerate(self.layers):
            if self.owner(i) != i:
                continue
            p = f"l{i}."
            sandwich = self.design.block == "sandwich"
            norm(p + "norm1")
            if sandwich:
                norm(p + "norm1b")
            t.update(s.mixer.tensor_shapes(p + "mix.", d))
            if s.mlp is not None:
                if self.design.block != "parallel":
                    norm(p + "norm2")
                if sandwich:
                    norm(p + "norm2b")
                t.update(s.mlp.tensor_shapes(p + "mlp.", d))
        norm("final.norm")
        if not self.design.tied:
            t["head"] = (self.vocab_size, d)
        return t

    def unused_tensors(self) -> set:
        """Names a checkpoint may hold although no layer reads them: the mixing share of a layer that does not mix, the
        second norm of a layer without a feed-forward."""
        out = set()
        if self.design.block in ("sandwich", "pre"):
            return {f"l{i}.{n}" for i, s in enumerate(self.layers) if s.mlp is None for n in ("norm2", "norm2b")}
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


def sandwich_layers(order: str, attention: dict, latent: dict, ff: int, moe: dict, dense: tuple = ()) -> tuple:
    """Layers of a Bikilix model: 'w' a windowed attention layer (`attention`), 'l' a latent one (`latent`); the layers whose index is in
    `dense` have a dense feed-forward of hidden size `ff`, the others routed experts (`moe`)."""
    design = DESIGNS["Bikilix"]

    def rot(m):
        return {**m, "rot": RotarySpec(**m["rot"])}
    mixers = {"w": AttentionSpec(**rot(attention), **{k: v for k, v in design.attention.items() if k != "sliding"}), "l": LatentSpec(**rot(latent))}
    return tuple(LayerSpec(mixers[c], DenseSpec(ff, design.act, design.gated) if i in dense else MoESpec(**moe, **design.experts))
                 for i, c in enumerate(order))


def prenorm_layers(order: str, attention: dict, left: dict, right: dict, scales: tuple, retention: dict, ff: int, moe: dict, dense: tuple = (),
                   kv_from: dict | None = None) -> tuple:
    """Layers of a Seredra model: 'a' an attention layer, 'p' a parallel one (`left`, `right`, `scales`), 'r' retention; the layers whose
    index is in `dense` have a dense feed-forward of hidden size `ff`, the others routed experts (`moe`); `kv_from`: attention layer ->
    the one whose keys and values it uses."""
    design = DESIGNS["Seredra"]

    def rot(m):
        return {**m, "rot": RotarySpec(**m["rot"], half=True)}

    def mixer(i, c):
        if c == "a":
            return AttentionSpec(**attention, **design.attention, kv_from=(kv_from or {}).get(i))
        if c == "r":
            return RetentionSpec(**rot(retention))
        return ParallelSpec(AttentionSpec(**rot(left), **{k: v for k, v in design.left.items() if k != "half"}), SelectiveSpec(**right), scales)
    return tuple(LayerSpec(mixer(i, c), DenseSpec(ff, design.act, design.gated) if i in dense else MoESpec(**moe, **design.experts))
                 for i, c in enumerate(order))
