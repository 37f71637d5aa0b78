"""Model configurations for the decoder-only families (GPT-2 style, Llama style, layered) and named presets."""
from __future__ import annotations

from dataclasses import dataclass, asdict

from .layered import LayeredConfig, LoopSpec, hybrid_layers, prenorm_layers, sandwich_layers, uniform_layers


@dataclass
class GPTConfig:
    """Decoder-only transformer.

    arch "gpt2": pre-LayerNorm, learned positions, GELU MLP, biases, tied input/output embedding.
    arch "llama": RMSNorm, rotary positions, grouped-query attention, SwiGLU MLP, no biases, untied head.
    """
    vocab_size: int = 50257
    seq_len: int = 1024
    n_layer: int = 12
    n_head: int = 12
    d_model: int = 768
    ffn_dim: int = 3072
    arch: str = "gpt2"
    n_kv_head: int = 0
    rope_theta: float = 500000.0
    norm_eps: float = 1e-5
    tie_embeddings: bool = True
    init_std: float = 0.02
    vocab_multiple: int = 128      # the embedding / head are padded to this multiple for aligned GEMM tiles

    def __post_init__(self):
        if self.n_kv_head == 0:
            self.n_kv_head = self.n_head
        if self.d_model % self.n_head or self.n_head % self.n_kv_head:
            raise ValueError("d_model % n_head and n_head % n_kv_head must both be 0")
        if self.arch not in ("gpt2", "llama"):
            raise ValueError(f"unknown arch {self.arch!r}")
        if self.arch == "llama":
            self.tie_embeddings = False

    @property
    def head_dim(self) -> int:
        return self.d_model // self.n_head

    @property
    def vocab_padded(self) -> int:
        m = self.vocab_multiple
        return (self.vocab_size + m - 1) // m * m

    @property
    def qkv_dim(self) -> int:
        return (self.n_head + 2 * self.n_kv_head) * self.head_dim

    def num_parameters(self, padded: bool = False) -> int:
        v = self.vocab_padded if padded else self.vocab_size
        d, f = self.d_model, self.ffn_dim
        if self.arch == "gpt2":
            per_layer = 2 * 2 * d + (self.qkv_dim * d + self.qkv_dim) + (d * d + d) + (f * d + f) + (d * f + d)
            return v * d + self.seq_len * d + self.n_layer * per_layer + 2 * d
        per_layer = 2 * d + self.qkv_dim * d + d * d + 2 * f * d + d * f
        return v * d + self.n_layer * per_layer + d + v * d

    def flops_per_token(self) -> float:
        """Training FLOPs per token: 6 x (matmul parameters) + causal attention."""
        d, f = self.d_model, self.ffn_dim
        mlp = (2 if self.arch == "gpt2" else 3) * f * d
        per_layer = self.qkv_dim * d + d * d + mlp
        matmul_params = self.n_layer * per_layer + self.vocab_padded * d
        attn = self.n_layer * 2 * self.seq_len * d      # QK^T and PV, causal half, per token, forward MACs*2/2
        return 6.0 * matmul_params + 3.0 * attn

    def to_dict(self) -> dict:
        return asdict(self)


PRESETS = {
    # tiny LM for the CPU reference backend
    "tiny-lm": dict(vocab_size=1024, seq_len=64, n_layer=2, n_head=4, d_model=128, ffn_dim=512, arch="gpt2",
                    tie_embeddings=False, vocab_multiple=1),
    # GPT-2 small: the headline training benchmark
    "gpt2-small": dict(vocab_size=50257, seq_len=1024, n_layer=12, n_head=12, d_model=768, ffn_dim=3072, arch="gpt2"),
    # Llama-style 8B: tensor / pipeline parallel training and serving
    "llama-8b": dict(vocab_size=128256, seq_len=4096, n_layer=32, n_head=32, n_kv_head=8, d_model=4096, ffn_dim=14336,
                     arch="llama", rope_theta=500000.0),
    # small shapes for tests
    "gpt2-test": dict(vocab_size=1000, seq_len=128, n_layer=2, n_head=4, d_model=256, ffn_dim=1024, arch="gpt2"),
    "llama-test": dict(vocab_size=1000, seq_len=128, n_layer=2, n_head=4, n_kv_head=2, d_model=256, ffn_dim=512,
                       arch="llama", rope_theta=10000.0),
    # layered decoders: `n_layer` equal layers of the given mixer and feed-forward
    "dolurax-test": dict(arch="Dolurax", vocab_size=1000, d_model=128, n_layer=3, seq_len=512, logit_scale=1.5, logit_softcap=20.0,
                         mixer=dict(heads=6, kv_heads=2, dim=48, vdim=32, scale=0.15, softcap=12.0, chunk=40, v_mix=True),
                         mlp=dict(ff=64, experts=12, top=3, groups=3, keep=2, shared_ff=40)),
    # one decoder layer about the size of a Llama-8B layer: same width, heads and head size, same feed-forward work per token
    # (7 routed experts + the shared one of 1792 = 14336)
    "dolurax-moe": dict(arch="Dolurax", vocab_size=128256, d_model=4096, n_layer=32, logit_scale=1.0, logit_softcap=30.0,
                        mixer=dict(heads=32, kv_heads=8, dim=128, vdim=128, scale=0.08838834764831845, softcap=30.0, chunk=8192,
                                   v_mix=True),
                        mlp=dict(ff=1792, experts=32, top=7, groups=4, keep=2, shared_ff=1792)),
    # layered decoders whose mixers carry state (order: p = attention beside a state-space mixer, d = delta rule)
    "vafodra-test": dict(arch="Vafodra", vocab_size=1000, d_model=128, seq_len=512, embed_scale=6.0, residual_mult=0.4, order="pdpd",
                         weights_of={2: 0},
                         left=dict(heads=6, kv_heads=2, dim=48, vdim=32, scale=0.15, window=40, keep_first=3),
                         right=dict(heads=4, vdim=40, state=24, groups=2, norm_groups=4, conv=3),
                         delta=dict(heads=6, kv_heads=3, dim=24, vdim=40, conv=4), ff=dict(p=192, d=256)),
    # about the size of a Llama-8B layer: same width, heads and head size, the feed-forward takes what the mixers leave of the
    # parameters
    "vafodra-8b": dict(arch="Vafodra", vocab_size=128256, d_model=4096, embed_scale=1.0, residual_mult=0.5, order="ppdp" * 8,
                       left=dict(heads=32, kv_heads=8, dim=128, vdim=128, scale=0.08838834764831845, window=2048, keep_first=4),
                       right=dict(heads=128, vdim=64, state=128, groups=8, norm_groups=8, conv=4),
                       delta=dict(heads=32, kv_heads=16, dim=128, vdim=128, conv=4), ff=dict(p=5376, d=12288)),
    # layered decoders with norms around every sublayer (order: w = windowed attention, l = latent attention); layers
    # loop.start .. loop.stop - 1 run several times
    "bikilix-test": dict(arch="Bikilix", vocab_size=1000, d_model=128, seq_len=512, embed_scale=2.0, order="wlwl", dense=(0,), ff=192,
                         loop=dict(start=1, stop=3, times=2),
                         attention=dict(heads=6, kv_heads=2, dim=48, vdim=32, scale=0.15, window=40, rot=dict(dims=16, base=10000.0)),
                         latent=dict(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=48, q_rank=56, scale=0.2,
                                     rot=dict(dims=16, base=20000.0, factor=4.0, original=128, fast=16.0, slow=1.0, scaled=True)),
                         moe=dict(ff=64, experts=12, top=3, groups=3, keep=2, limit=2.0)),
    # about the size of Llama-8B layers: same width and heads; a third of the layers run twice
    "bikilix-moe": dict(arch="Bikilix", vocab_size=128256, d_model=4096, order="wwl" * 8, dense=(0,), ff=14336,
                        loop=dict(start=6, stop=14, times=2),
                        attention=dict(heads=32, kv_heads=8, dim=128, vdim=128, scale=0.08838834764831845, window=2048,
                                       rot=dict(dims=64, base=500000.0)),
                        latent=dict(heads=32, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=1536, scale=0.07216878364870322,
                                    rot=dict(dims=64, base=500000.0, factor=8.0, original=4096, fast=32.0, slow=1.0, scaled=True)),
                        moe=dict(ff=2048, experts=32, top=7, groups=4, keep=2, limit=7.0)),
    # layered decoders with a norm in front of every sublayer (order: p = attention beside a selective scan, r = retention, a = attention
    # with short convolutions; kv_from: an attention layer -> the one whose keys and values it uses)
    "seredra-test": dict(arch="Seredra", vocab_size=1000, d_model=128, seq_len=512, embed_scale=3.0, order="rapa", kv_from={3: 1}, dense=(1, 2),
                         attention=dict(heads=6, kv_heads=2, dim=48, vdim=32, scale=0.15, conv=3, temp_coef=0.3, temp_every=40),
                         left=dict(heads=3, kv_heads=1, dim=40, vdim=40, scale=0.16, softcap=15.0,
                                   rot=dict(dims=32, base=10000.0, factor=4.0, original=128, fast=16.0, slow=1.0, scaled=True)),
                         right=dict(inner=160, state=12, dt_rank=8, conv=4), scales=(0.8, 1.1),
                         retention=dict(heads=3, dim=24, vdim=56, decay=(0.9, 0.97, 0.995), rot=dict(dims=24, base=100000.0)), ff=192,
                         moe=dict(ff=64, experts=12, top=3)),
    # about the size of Llama-8B layers: same width, heads and head size; every third layer an attention layer, every other of them
    # without a cache of its own
    "seredra-moe": dict(arch="Seredra", vocab_size=128256, d_model=4096, embed_scale=1.0, order="pra" * 10, kv_from={i: i - 3 for i in range(5, 30, 6)},
                        dense=tuple(range(0, 30, 2)),
                        attention=dict(heads=32, kv_heads=8, dim=128, vdim=128, scale=0.08838834764831845, conv=4, temp_coef=0.1, temp_every=8192),
                        left=dict(heads=32, kv_heads=8, dim=128, vdim=128, scale=0.08838834764831845, softcap=50.0,
                                  rot=dict(dims=128, base=500000.0, factor=8.0, original=8192, fast=32.0, slow=1.0, scaled=True)),
                        right=dict(inner=8192, state=16, dt_rank=256, conv=4), scales=(1.0, 1.0),
                        retention=dict(heads=32, dim=128, vdim=256, decay=tuple(1.0 - 2.0 ** (-5 - 7 * i / 31) for i in range(32)),
                                       rot=dict(dims=128, base=10000.0)), ff=14336, moe=dict(ff=2048, experts=32, top=5)),
}


def preset(name: str, **overrides):
    cfg = dict(PRESETS[name])
    cfg.update(overrides)
    if "order" in cfg:
        if "n_layer" in cfg:
            cfg["order"] = (cfg["order"] * cfg["n_layer"])[:cfg.pop("n_layer")]
        if cfg["arch"] == "Bikilix":
            n, loop = len(cfg["order"]), cfg.pop("loop", None)
            cfg["layers"] = sandwich_layers(*(cfg.pop(k) for k in ("order", "attention", "latent", "ff", "moe")), cfg.pop("dense", ()))
            if loop and loop["start"] < n:
                cfg["loop"] = LoopSpec(loop["start"], min(loop["stop"], n), loop["times"])
            return LayeredConfig(**cfg)
        if cfg["arch"] == "Seredra":
            keep = {i: j for i, j in cfg.pop("kv_from", {}).items() if i < len(cfg["order"]) and cfg["order"][i] == cfg["order"][j] == "a"}
            cfg["layers"] = prenorm_layers(*(cfg.pop(k) for k in ("order", "attention", "left", "right", "scales", "retention", "ff", "moe")),
                                           cfg.pop("dense", ()), keep)
            return LayeredConfig(**cfg)
        cfg["layers"] = hybrid_layers(*(cfg.pop(k) for k in ("order", "left", "right", "delta", "ff")), cfg.pop("weights_of", None))
        return LayeredConfig(**cfg)
    if "mixer" in cfg:
        cfg["layers"] = uniform_layers(cfg.pop("n_layer"), cfg.pop("mixer"), cfg.pop("mlp"))
        return LayeredConfig(**cfg)
    return GPTConfig(**cfg)
