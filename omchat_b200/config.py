"""Configuration objects mirroring the reference's config surface.

`OmChatQwen2Config` keeps the attribute names the reference reads with getattr on the hot path (omchat_arch.py:25-28,
100,161,176; internVIT_encoder.py:16-17) and adds three knobs whose defaults reproduce reference behaviour:
`mm_pixel_shuffle_ratio` (1.0 = none), `kv_page_size`, `tp_size`.
"""
from __future__ import annotations

from dataclasses import dataclass, field, asdict
from typing import List, Optional

IMAGE_TOKEN_INDEX = -200  # omchat/constants.py:8
IGNORE_INDEX = -100


@dataclass
class InternVisionConfig:
    """intern_vit_6b/configuration_intern_vit.py:63-83 defaults (InternViT-6B-448px-V1-5)."""
    num_channels: int = 3
    patch_size: int = 14
    image_size: int = 448
    qkv_bias: bool = False
    hidden_size: int = 3200
    num_attention_heads: int = 25
    intermediate_size: int = 12800
    qk_normalization: bool = True
    num_hidden_layers: int = 45
    hidden_act: str = "gelu"
    layer_norm_eps: float = 1e-6
    initializer_factor: float = 0.1
    norm_type: str = "rms_norm"  # 'layer_norm' for the InternViT-300M variant (intern_vit_300m/modeling_intern_vit.py:61-64)

    def __post_init__(self):
        if self.norm_type not in ("rms_norm", "layer_norm"):
            raise ValueError(f"unknown norm_type {self.norm_type!r}")

    @classmethod
    def intern_vit_300m(cls, **overrides) -> "InternVisionConfig":
        """intern_vit_300m/configuration_intern_vit.py:60-80 defaults: the lighter tower (LayerNorm, no QK-norm, 16 heads of 64)."""
        kw = dict(hidden_size=1024, num_attention_heads=16, intermediate_size=4096, qk_normalization=False, num_hidden_layers=24,
                  norm_type="layer_norm", initializer_factor=1.0)
        kw.update(overrides)
        return cls(**kw)

    @property
    def num_patches(self) -> int:
        return (self.image_size // self.patch_size) ** 2

    @property
    def head_dim(self) -> int:
        return self.hidden_size // self.num_attention_heads


@dataclass
class OmChatQwen2Config:
    """omchat_qwen2.py:16-19 (Qwen2Config fields + the mm_* attributes); defaults = Qwen2-7B + InternViT-6B."""
    model_type: str = "omchat_qwen2"
    vocab_size: int = 152064
    hidden_size: int = 3584
    intermediate_size: int = 18944
    num_hidden_layers: int = 28
    num_attention_heads: int = 28
    num_key_value_heads: int = 4
    rms_norm_eps: float = 1e-6
    rope_theta: float = 1e6
    max_position_embeddings: int = 32768
    # multimodal attributes read by the reference
    mm_vision_tower: Optional[str] = "InternViT-6B-448px-V1-5"
    mm_projector_type: str = "mlp2x_gelu"
    mm_hidden_size: int = 3200
    mm_vision_select_layer: int = -1
    mm_vision_select_feature: str = "patch"
    delay_load: bool = False
    image_grid_pinpoints: List[List[int]] = field(default_factory=lambda: [
        [448, 896], [896, 448], [896, 896], [1344, 448], [448, 1344], [1344, 1344]])
    tokenizer_model_max_length: Optional[int] = None
    tokenizer_padding_side: str = "right"
    tune_mm_mlp_adapter: bool = False
    mm_use_im_start_end: bool = False
    eos_token_id: int = 151645
    pad_token_id: int = 151643
    # build-specific knobs (defaults reproduce the reference)
    mm_pixel_shuffle_ratio: float = 1.0
    kv_page_size: int = 64
    tp_size: int = 1
    vision_config: InternVisionConfig = field(default_factory=InternVisionConfig)

    def __post_init__(self):
        # build_vision_tower (multimodal_encoder/builder.py:11-14) picks the tower class from the NAME: a config that names the
        # 300M tower and leaves vision_config at the 6B defaults gets the 300M defaults
        name = (self.mm_vision_tower or "").lower()
        if "internvit-300m" in name and self.vision_config == InternVisionConfig():
            self.vision_config = InternVisionConfig.intern_vit_300m()
            if self.mm_hidden_size == 3200:
                self.mm_hidden_size = self.vision_config.hidden_size

    @property
    def head_dim(self) -> int:
        return self.hidden_size // self.num_attention_heads

    @property
    def pixel_shuffle_down(self) -> int:
        d = round(1.0 / self.mm_pixel_shuffle_ratio)
        if d < 1 or abs(1.0 / d - self.mm_pixel_shuffle_ratio) > 1e-6:
            raise ValueError(f"mm_pixel_shuffle_ratio must be 1/k, got {self.mm_pixel_shuffle_ratio}")
        return d

    @property
    def image_tokens_per_crop(self) -> int:
        g = self.vision_config.image_size // self.vision_config.patch_size
        return (g // self.pixel_shuffle_down) ** 2

    def to_dict(self):
        return asdict(self)


@dataclass
class OmChatQwen2MoeConfig(OmChatQwen2Config):
    """omchat_qwen2_moe.py:14-17: transformers Qwen2MoeConfig fields + the mm_* attributes. Defaults = Qwen1.5-MoE-A2.7B's
    language model (Qwen2MoeConfig defaults) under the same vision tower."""
    model_type: str = "omchat_qwen2_moe"
    hidden_size: int = 2048
    intermediate_size: int = 5632
    num_hidden_layers: int = 24
    num_attention_heads: int = 16
    num_key_value_heads: int = 16
    num_experts: int = 60
    num_experts_per_tok: int = 4
    moe_intermediate_size: int = 1408
    shared_expert_intermediate_size: int = 5632
    norm_topk_prob: bool = False
    decoder_sparse_step: int = 1
    mlp_only_layers: List[int] = field(default_factory=list)

    def layer_is_sparse(self, li: int) -> bool:
        """Qwen2MoeDecoderLayer.__init__ (transformers modeling_qwen2_moe.py:381-386)."""
        return li not in self.mlp_only_layers and self.num_experts > 0 and (li + 1) % self.decoder_sparse_step == 0


# ---------------------------------------------------------------------------------------------------------------------------
# Voduzen: a decoder-only language model described by a per-layer list (config.json: architecture "Voduzen").


@dataclass
class RotarySpec:
    """Pairwise-interleaved rotary embedding on the first `dims` dimensions of a vector: pair i = (2i, 2i + 1) turns by
    position * f_i, f_i = base^(-2i/dims). `scaling` (factor, original, fast, slow) blends f_i towards f_i / factor over a
    linear ramp in i and multiplies cos and sin by 0.1 ln(factor) + 1 (the constants 0.1 and 0.001 are fixed by the design).
    halves: pair i is (i, i + dims / 2) instead."""
    dims: int
    base: float
    scaling: Optional[dict] = None
    halves: bool = False

    def frequencies(self):
        """(f [dims / 2] as Python floats, multiplier of cos / sin) in double precision."""
        import math
        half = self.dims // 2
        f = [self.base ** (-2.0 * i / self.dims) for i in range(half)]
        mult = 1.0
        sc = self.scaling
        if sc:
            factor, orig = float(sc["factor"]), float(sc["original"])

            def turn_dim(turns: float) -> float:
                return self.dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))
            lo = max(math.floor(turn_dim(float(sc["fast"]))), 0)
            hi = min(math.ceil(turn_dim(float(sc["slow"]))), self.dims - 1)
            span = max(hi - lo, 0.001)
            for i in range(half):
                ramp = min(max((i - lo) / span, 0.0), 1.0)
                f[i] = f[i] / factor * ramp + f[i] * (1.0 - ramp)
            mult = 0.1 * math.log(factor) + 1.0
        return f, mult


@dataclass
class LatentAttentionSpec:
    """Attention whose keys and values are up-projections of a cached latent of width kv_rank plus one rotated key part of
    width rot_dim shared by the heads. q_rank: queries go through a normed latent of that width (None: one projection).
    sink: the softmax denominator has one more learned term per head. window: keys a row sees behind itself, itself included
    (None: all). head_gate: every head's output is multiplied by a sigmoid of a projection of the mixer's input; out_gate: every
    element of the concatenated heads is. kv_from: the layer whose cached rows this one attends to (it projects no keys or values of its own and caches nothing)."""
    heads: int
    dim: int        # unrotated query / key dimensions per head
    rot_dim: int    # rotated query / key dimensions per head
    vdim: int
    kv_rank: int
    scale: float
    rot: RotarySpec = None
    q_rank: Optional[int] = None
    sink: bool = False
    window: Optional[int] = None
    head_gate: bool = False
    kv_from: Optional[int] = None
    out_gate: bool = False


@dataclass
class RouterMoeSpec:
    """Mixture of experts: `experts` feed-forward experts (relu^2, no biases) of width expert_ff followed by `identity`
    identity outputs of the router; every token uses `top` of them; shared_ff: width of the always-on expert (None: none)."""
    experts: int
    identity: int
    top: int
    expert_ff: int
    shared_ff: Optional[int] = None


@dataclass
class VoduzenLayerSpec:
    type: str
    mixer: LatentAttentionSpec
    mlp: Optional[RouterMoeSpec]


@dataclass
class VoduzenConfig:
    model_type: str = "voduzen"
    vocab_size: int = 0
    hidden_size: int = 0
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    norm_eps: float = 1e-6
    layers: List[VoduzenLayerSpec] = field(default_factory=list)
    kv_page_size: int = 64       # engine knob: tokens per cache page
    eos_token_id: int = -1
    pad_token_id: int = 0

    MIXERS = ("latent_attention", "latent_attention_2")

    @classmethod
    def from_dict(cls, d: dict) -> "VoduzenConfig":
        layers = []
        for i, ld in enumerate(d["layers"]):
            typ = ld["type"]
            if typ not in cls.MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {typ!r}")
            m = ld["mixer"]
            rot = m.get("rot") or {}
            rspec = RotarySpec(dims=int(rot.get("dims", m.get("rot_dim", 0))), base=float(rot.get("base", 10000.0)),
                               scaling=dict(rot["scaling"]) if rot.get("scaling") else None)
            if rspec.dims > int(m["rot_dim"]) or rspec.dims % 2:
                raise ValueError(f"layer {i}: rot.dims must be even and at most rot_dim")
            # the first kind projects queries directly and has a sink; the second sends queries through a latent, plain softmax
            mix = LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                                      kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot=rspec,
                                      q_rank=int(m["q_rank"]) if typ == "latent_attention_2" else None,
                                      sink=typ == "latent_attention")
            mlp = None
            md = ld.get("mlp")
            if md:
                if md.get("kind", "moe") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {md.get('kind')!r}")
                r = md["router"]
                sh = md.get("shared")
                mlp = RouterMoeSpec(experts=int(r["experts"]), identity=int(r.get("identity", 0)), top=int(r["top"]),
                                    expert_ff=int(md["expert"]["ff"]), shared_ff=int(sh["ff"]) if sh else None)
            layers.append(VoduzenLayerSpec(type=typ, mixer=mix, mlp=mlp))
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]),
                   embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                   logit_scale=float(d.get("logit_scale", 1.0)), norm_eps=float((d.get("norm") or {}).get("eps", 1e-6)),
                   layers=layers, kv_page_size=int(d.get("kv_page_size", 64)), eos_token_id=int(d.get("eos_token_id", -1)),
                   pad_token_id=int(d.get("pad_token_id", 0)))

    def to_dict(self) -> dict:
        """The config.json form (round-trips through from_dict)."""
        out_layers = []
        for l in self.layers:
            m = l.mixer
            rot = {"base": m.rot.base, "dims": m.rot.dims}
            if m.rot.scaling:
                rot["scaling"] = dict(m.rot.scaling)
            md = {"dim": m.dim, "heads": m.heads, "kv_rank": m.kv_rank, "rot": rot, "rot_dim": m.rot_dim, "scale": m.scale,
                  "vdim": m.vdim}
            if m.q_rank is not None:
                md["q_rank"] = m.q_rank
            mlp = None
            if l.mlp is not None:
                mlp = {"kind": "moe", "expert": {"ff": l.mlp.expert_ff},
                       "router": {"experts": l.mlp.experts, "identity": l.mlp.identity, "top": l.mlp.top},
                       "shared": {"ff": l.mlp.shared_ff} if l.mlp.shared_ff else None}
            out_layers.append({"type": l.type, "mixer": md, "mlp": mlp})
        return {"architecture": "Voduzen", "vocab": self.vocab_size, "width": self.hidden_size,
                "embedding": {"scale": self.embedding_scale}, "logit_scale": self.logit_scale, "norm": {"eps": self.norm_eps},
                "layers": out_layers, "kv_page_size": self.kv_page_size, "eos_token_id": self.eos_token_id,
                "pad_token_id": self.pad_token_id}


# --------------------------------------------------------------------------------------------------------------------- Tifisun
@dataclass
class DeltaRuleSpec:
    """Gated delta rule: a [dim, vdim] fp32 state per head, decayed, corrected towards the new value along the key, read by the
    query. kv_heads query / key heads serve heads value heads. conv: taps of the causal per-channel convolution in front of
    q, k, v. channel_decay: one decay per key channel (projected through `decay_rank` columns) instead of one per head;
    gate_rank: the output gate is projected through that many columns and squashed by a sigmoid (None: one projection, silu)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    channel_decay: bool = False
    decay_rank: Optional[int] = None
    gate_rank: Optional[int] = None


@dataclass
class WindowAttentionSpec:
    """Softmax attention over a sliding window of `window` keys (the row's own included), grouped heads, no rotation. Queries and
    keys are RMS-normed over their whole projection; scores are scaled, soft-capped (softcap * tanh(s / softcap); 0 = off) and
    get a learned bias by distance: `bias_rows` table rows, the first half one per distance, the rest logarithmic up to bias_max."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    softcap: float = 0.0
    bias_max: float = 0.0

    @staticmethod
    def bucket(n: int, rows: int, far: float) -> int:
        import math
        half = rows // 2
        if n < half:
            return n
        if half < 1 or far <= half:      # no logarithmic range to spread over: everything further shares the last row
            return rows - 1
        return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))


@dataclass
class DecayAttentionSpec:
    """Linear attention with one constant decay per head: S <- decay_h S + k v^T, o = S^T q, silu on q, k, v."""
    heads: int
    dim: int
    vdim: int
    decay: List[float] = field(default_factory=list)


@dataclass
class ParallelMixerSpec:
    left: WindowAttentionSpec
    right: DecayAttentionSpec


@dataclass
class DenseMlpSpec:
    """act(W_gate x + b) * (W_up x + b) -> W_down + b, act = tanh-form gelu (bias False: no b)."""
    ff: int
    bias: bool = True


@dataclass
class TifisunLayerSpec:
    type: str                      # 'delta' | 'channel_delta' | 'parallel'
    mixer: object                  # DeltaRuleSpec | ParallelMixerSpec
    mlp: Optional[DenseMlpSpec]
    weights_of: Optional[int] = None   # the layer whose tensors this one uses (its cache and state are its own)



@dataclass
class TifisunConfig:
    model_type: str = "tifisun"
    vocab_size: int = 0
    hidden_size: int = 0
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    norm_eps: float = 1e-6
    layers: List[TifisunLayerSpec] = field(default_factory=list)
    kv_page_size: int = 64       # engine knob: tokens per cache page
    eos_token_id: int = -1
    pad_token_id: int = 0

    MIXERS = ("delta", "channel_delta", "parallel")

    @classmethod
    def from_dict(cls, d: dict) -> "TifisunConfig":
        layers = []
        for i, ld in enumerate(d["layers"]):
            typ, m = ld["type"], ld["mixer"]
            if typ not in cls.MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {typ!r}")
            if typ == "parallel":
                l, r = m["left"], m["right"]
                left = WindowAttentionSpec(heads=int(l["heads"]), kv_heads=int(l.get("kv_heads", l["heads"])), dim=int(l["dim"]),
                                           vdim=int(l["vdim"]), scale=float(l["scale"]), window=int(l["mask"]["size"]),
                                           softcap=float(l.get("softcap") or 0.0), bias_max=float(l.get("bias_max") or 0.0))
                right = DecayAttentionSpec(heads=int(r["heads"]), dim=int(r["dim"]), vdim=int(r["vdim"]),
                                           decay=[float(x) for x in r["decay"]])
                if left.heads % left.kv_heads or len(right.decay) != right.heads or left.window < 1:
                    raise ValueError(f"layer {i}: inconsistent mixer sizes")
                mix = ParallelMixerSpec(left, right)
            else:
                mix = DeltaRuleSpec(heads=int(m["heads"]), kv_heads=int(m.get("kv_heads", m["heads"])), dim=int(m["dim"]),
                                    vdim=int(m["vdim"]), conv=int(m["conv"]), channel_decay=typ == "channel_delta",
                                    decay_rank=int(m["decay_rank"]) if m.get("decay_rank") else None,
                                    gate_rank=int(m["gate_rank"]) if m.get("gate_rank") else None)
                if mix.heads % mix.kv_heads or mix.conv < 1:
                    raise ValueError(f"layer {i}: inconsistent mixer sizes")
            md = ld.get("mlp")
            if md and md.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {md.get('kind')!r}")
            wo = ld.get("weights_of")
            if wo is not None and not (0 <= int(wo) < len(d["layers"]) and int(wo) != i and d["layers"][int(wo)]["type"] == typ):
                raise ValueError(f"layer {i}: weights_of must name another layer of the same type")
            layers.append(TifisunLayerSpec(type=typ, mixer=mix, mlp=DenseMlpSpec(ff=int(md["ff"])) if md else None,
                                           weights_of=int(wo) if wo is not None else None))
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]),
                   embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                   residual_mult=float(d.get("residual_mult", 1.0)), norm_eps=float((d.get("norm") or {}).get("eps", 1e-6)),
                   layers=layers, kv_page_size=int(d.get("kv_page_size", 64)), eos_token_id=int(d.get("eos_token_id", -1)),
                   pad_token_id=int(d.get("pad_token_id", 0)))

    def to_dict(self) -> dict:
        """The config.json form (round-trips through from_dict)."""
        out = []
        for l in self.layers:
            if l.type == "parallel":
                a, b = l.mixer.left, l.mixer.right
                md = {"left": {"bias_max": a.bias_max, "dim": a.dim, "heads": a.heads, "kv_heads": a.kv_heads,
                               "mask": {"size": a.window}, "scale": a.scale, "softcap": a.softcap, "vdim": a.vdim},
                      "right": {"decay": list(b.decay), "dim": b.dim, "heads": b.heads, "vdim": b.vdim}}
            else:
                m = l.mixer
                md = {"conv": m.conv, "dim": m.dim, "heads": m.heads, "kv_heads": m.kv_heads, "vdim": m.vdim}
            e = {"type": l.type, "mixer": md, "mlp": {"ff": l.mlp.ff, "kind": "dense"} if l.mlp else None}
            if l.weights_of is not None:
                e["weights_of"] = l.weights_of
            out.append(e)
        return {"architecture": "Tifisun", "vocab": self.vocab_size, "width": self.hidden_size,
                "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult, "norm": {"eps": self.norm_eps},
                "layers": out, "kv_page_size": self.kv_page_size, "eos_token_id": self.eos_token_id,
                "pad_token_id": self.pad_token_id}


# --------------------------------------------------------------------------------------------------------------------- Fofisun
@dataclass
class DiffAttentionSpec:
    """Differential softmax attention without rotation: every head has two score maps (queries and keys of their own, `dim` wide)
    over one set of values; o = a1 - lambda a2, RMS-normed over the head and scaled by 1 - diff, lambda = exp(lq1 . lk1) -
    exp(lq2 . lk2) + diff. conv: taps of the causal per-channel convolution behind the q, k, v projections (0: none). Queries and
    keys are RMS-normed per head and map. window: keys a row sees behind itself, itself included (None: all); keep_first: the
    first keys of the sequence stay visible behind the window. The concatenated heads pass a sigmoid gate."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    window: Optional[int] = None
    keep_first: int = 0
    conv: int = 0


@dataclass
class GeluMlpSpec:
    """W_down gelu(W_up x) with the erf form of gelu, no biases."""
    ff: int


@dataclass
class ClampedMoeSpec:
    """`experts` gated experts of width expert_ff, `top` per token chosen by the router's logits (weights: softmax over the chosen
    logits alone). An expert: g = min(W_gate x, limit), u = clamp(W_up x, -limit, limit), W_down (g sigmoid(1.702 g) (u + 1)).
    shared_ff: width of an expert that every token passes, scaled by a sigmoid gate of the token (None: none)."""
    experts: int
    top: int
    expert_ff: int
    limit: float
    shared_ff: Optional[int] = None
    shared_limit: float = 0.0


@dataclass
class FofisunLayerSpec:
    type: str                      # 'attention'
    mixer: DiffAttentionSpec
    mlp: object                    # GeluMlpSpec | ClampedMoeSpec | None


@dataclass
class FofisunConfig:
    model_type: str = "fofisun"
    vocab_size: int = 0
    hidden_size: int = 0
    norm_eps: float = 1e-6
    layers: List[FofisunLayerSpec] = field(default_factory=list)
    loop_start: int = 0            # layers loop_start .. loop_stop - 1 run loop_times times in a row (the same tensors, a cache per run)
    loop_stop: int = 0
    loop_times: int = 1
    kv_page_size: int = 64         # engine knob: tokens per cache page
    eos_token_id: int = -1
    pad_token_id: int = 0

    MIXERS = ("attention",)
    POSITION_BASE = 10000.0        # sinusoidal position vectors: entry 2i / 2i + 1 = sin / cos(p * base^(-2i / width))
    SWISH_SLOPE = 1.702            # the experts' gate is g * sigmoid(SWISH_SLOPE * g)
    UP_SHIFT = 1.0                 # ... times (u + UP_SHIFT)

    def layer_runs(self) -> List[int]:
        """The layer index of every layer run, in execution order."""
        n = len(self.layers)
        if self.loop_stop <= self.loop_start:
            return list(range(n))
        return list(range(self.loop_start)) + list(range(self.loop_start, self.loop_stop)) * self.loop_times + list(range(self.loop_stop, n))

    @classmethod
    def from_dict(cls, d: dict) -> "FofisunConfig":
        layers = []
        for i, ld in enumerate(d["layers"]):
            typ, m = ld["type"], ld["mixer"]
            if typ not in cls.MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {typ!r}")
            mask = m.get("mask") or {}
            mix = DiffAttentionSpec(heads=int(m["heads"]), kv_heads=int(m.get("kv_heads") or m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                    scale=float(m["scale"]), diff=float(m["diff"]),
                                    window=int(mask["size"]) if mask.get("size") is not None else None,
                                    keep_first=int(mask.get("keep_first") or 0), conv=int(m.get("conv") or 0))
            if mix.heads < 1 or mix.kv_heads < 1 or mix.heads % mix.kv_heads or mix.conv < 0 or mix.keep_first < 0 or \
                    (mix.window is not None and mix.window < 1):
                raise ValueError(f"layer {i}: inconsistent mixer sizes")
            md, mlp = ld.get("mlp"), None
            if md:
                kind = md.get("kind", "dense")
                if kind == "dense":
                    mlp = GeluMlpSpec(ff=int(md["ff"]))
                elif kind == "moe":
                    r, e, sh = md["router"], md["expert"], md.get("shared")
                    mlp = ClampedMoeSpec(experts=int(r["experts"]), top=int(r["top"]), expert_ff=int(e["ff"]), limit=float(e["limit"]),
                                         shared_ff=int(sh["ff"]) if sh else None, shared_limit=float(sh["limit"]) if sh else 0.0)
                    if not 1 <= mlp.top <= mlp.experts:
                        raise ValueError(f"layer {i}: top must be between 1 and the number of experts")
                else:
                    raise ValueError(f"layer {i}: unknown feed-forward kind {kind!r}")
            layers.append(FofisunLayerSpec(type=typ, mixer=mix, mlp=mlp))
        lp = d.get("loop") or {}
        start, stop, times = int(lp.get("start", 0)), int(lp.get("stop", 0)), int(lp.get("times", 1))
        if lp and not (0 <= start <= stop <= len(layers) and times >= 1):
            raise ValueError("loop: start <= stop within the layers and times >= 1 are required")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), norm_eps=float((d.get("norm") or {}).get("eps", 1e-6)),
                   layers=layers, loop_start=start, loop_stop=stop, loop_times=times, kv_page_size=int(d.get("kv_page_size", 64)),
                   eos_token_id=int(d.get("eos_token_id", -1)), pad_token_id=int(d.get("pad_token_id", 0)))

    def to_dict(self) -> dict:
        """The config.json form (round-trips through from_dict)."""
        out = []
        for l in self.layers:
            m = l.mixer
            md = {"conv": m.conv, "diff": m.diff, "dim": m.dim, "heads": m.heads, "kv_heads": m.kv_heads,
                  "mask": {"keep_first": m.keep_first, "size": m.window}, "scale": m.scale, "vdim": m.vdim}
            if isinstance(l.mlp, GeluMlpSpec):
                mlp = {"ff": l.mlp.ff, "kind": "dense"}
            elif isinstance(l.mlp, ClampedMoeSpec):
                s = l.mlp
                mlp = {"expert": {"ff": s.expert_ff, "limit": s.limit}, "kind": "moe", "router": {"experts": s.experts, "top": s.top},
                       "shared": {"ff": s.shared_ff, "limit": s.shared_limit} if s.shared_ff else None}
            else:
                mlp = None
            out.append({"type": l.type, "mixer": md, "mlp": mlp})
        return {"architecture": "Fofisun", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
                "layers": out, "loop": {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times},
                "kv_page_size": self.kv_page_size, "eos_token_id": self.eos_token_id, "pad_token_id": self.pad_token_id}


# --------------------------------------------------------------------------------------------------------------------- Vefunex
@dataclass
class SoftmaxAttentionSpec:
    """Causal softmax attention over all earlier keys with grouped heads. Which of the optional mechanisms a layer has:
    rot (RotarySpec or None): pairwise-interleaved rotation of the first rot.dims dimensions of queries and keys; q_temp_coef /
    q_temp_every: queries are multiplied by 1 + coef ln(floor((p + 1) / every) + 1) at position p (coef 0: off); value_norm: every
    head's value is divided by its root mean square before it is cached; softcap: scores become softcap tanh(score / softcap)
    (0: off); sink: one more learned term exp(sink_h) per head in the softmax denominator; gate: the concatenated heads are
    multiplied by a sigmoid of a projection of the mixer's input."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotarySpec] = None
    q_temp_coef: float = 0.0
    q_temp_every: int = 1
    value_norm: bool = False
    softcap: float = 0.0
    sink: bool = False
    gate: bool = False


@dataclass
class SelectiveScanSpec:
    """Selective state-space mixer: `inner` channels with `state` fp32 states each, a causal convolution of `conv` taps (with bias)
    and silu in front, step sizes through a projection of rank dt_rank; S <- exp(dt A) S + dt x B, y = S C + D x, gated by silu(z)."""
    inner: int
    state: int
    dt_rank: int
    conv: int


@dataclass
class AttentionScanMixerSpec:
    """Two mixers side by side on the same input: left_scale * attention + right_scale * selective scan."""
    left: SoftmaxAttentionSpec
    right: SelectiveScanSpec
    left_scale: float = 1.0
    right_scale: float = 1.0


@dataclass
class GatedLinearAttentionSpec:
    """Gated linear attention: per head S <- diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t with one decay per key channel,
    alpha = sigmoid(low-rank projection + bias)^(1 / tau); queries scaled by dim^-1/2; the read-out is RMS-normed per head and gated
    by silu of a projection."""
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass
class SigmoidMoeSpec:
    """`experts` gated experts (silu, no biases) of width expert_ff; every token uses the `top` experts with the largest sigmoid
    router scores; the scores are used as they are and multiply the experts' INPUT."""
    experts: int
    top: int
    expert_ff: int


@dataclass
class VefunexLayerSpec:
    type: str                      # 'attention' | 'parallel' | 'gla'
    mixer: object                  # SoftmaxAttentionSpec | AttentionScanMixerSpec | GatedLinearAttentionSpec
    mlp: Optional[SigmoidMoeSpec]


@dataclass
class VefunexConfig:
    model_type: str = "vefunex"
    vocab_size: int = 0
    hidden_size: int = 0
    norm_eps: float = 1e-6
    residual_mult: float = 1.0
    logit_softcap: float = 0.0     # logits become cap * tanh(logits / cap) (0: off)
    canon_taps: int = 1            # taps of the convolution every sublayer's input passes (h + conv(h))
    layers: List[VefunexLayerSpec] = field(default_factory=list)
    kv_page_size: int = 64         # engine knob: tokens per cache page
    eos_token_id: int = -1
    pad_token_id: int = 0

    MIXERS = ("attention", "parallel", "gla")

    @staticmethod
    def _attention(m: dict, i: int, *, value_norm: bool, sink: bool, gate: bool) -> SoftmaxAttentionSpec:
        rot, qt = m.get("rot"), m.get("q_temp")
        spec = SoftmaxAttentionSpec(heads=int(m["heads"]), kv_heads=int(m.get("kv_heads") or m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                    scale=float(m["scale"]), rot=RotarySpec(dims=int(rot["dims"]), base=float(rot["base"])) if rot else None,
                                    q_temp_coef=float(qt["coef"]) if qt else 0.0, q_temp_every=int(qt["every"]) if qt else 1,
                                    value_norm=value_norm, softcap=float(m.get("softcap") or 0.0), sink=sink, gate=gate)
        if spec.heads < 1 or spec.kv_heads < 1 or spec.heads % spec.kv_heads or spec.q_temp_every < 1 or \
                (spec.rot is not None and (spec.rot.dims % 2 or not 0 <= spec.rot.dims <= spec.dim)):
            raise ValueError(f"layer {i}: inconsistent attention sizes")
        return spec

    @classmethod
    def from_dict(cls, d: dict) -> "VefunexConfig":
        layers = []
        for i, ld in enumerate(d["layers"]):
            typ, m = ld["type"], ld["mixer"]
            if typ == "attention":
                mix = cls._attention(m, i, value_norm=True, sink=False, gate=False)
            elif typ == "parallel":
                r = m["right"]
                right = SelectiveScanSpec(inner=int(r["inner"]), state=int(r["state"]), dt_rank=int(r["dt_rank"]), conv=int(r["conv"]))
                if min(right.inner, right.state, right.dt_rank, right.conv) < 1:
                    raise ValueError(f"layer {i}: inconsistent selective-scan sizes")
                mix = AttentionScanMixerSpec(left=cls._attention(m["left"], i, value_norm=False, sink=True, gate=True), right=right,
                                             left_scale=float(m.get("left_scale", 1.0)), right_scale=float(m.get("right_scale", 1.0)))
            elif typ == "gla":
                mix = GatedLinearAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), tau=float(m["tau"]))
                if min(mix.heads, mix.dim, mix.vdim) < 1 or not mix.tau > 0:
                    raise ValueError(f"layer {i}: inconsistent gated-linear-attention sizes")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {typ!r}")
            md, mlp = ld.get("mlp"), None
            if md:
                if md.get("kind", "moe") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {md.get('kind')!r}")
                mlp = SigmoidMoeSpec(experts=int(md["router"]["experts"]), top=int(md["router"]["top"]), expert_ff=int(md["expert"]["ff"]))
                if not 1 <= mlp.top <= mlp.experts or mlp.expert_ff < 1:
                    raise ValueError(f"layer {i}: top must be between 1 and the number of experts")
            layers.append(VefunexLayerSpec(type=typ, mixer=mix, mlp=mlp))
        taps = int((d.get("canon") or {}).get("taps", 1))
        if taps < 1:
            raise ValueError("canon.taps must be at least 1")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), norm_eps=float((d.get("norm") or {}).get("eps", 1e-6)),
                   residual_mult=float(d.get("residual_mult", 1.0)), logit_softcap=float(d.get("logit_softcap") or 0.0), canon_taps=taps,
                   layers=layers, kv_page_size=int(d.get("kv_page_size", 64)), eos_token_id=int(d.get("eos_token_id", -1)),
                   pad_token_id=int(d.get("pad_token_id", 0)))

    def to_dict(self) -> dict:
        """The config.json form (round-trips through from_dict)."""
        def att(a: SoftmaxAttentionSpec) -> dict:
            md = {"dim": a.dim, "heads": a.heads, "kv_heads": a.kv_heads, "scale": a.scale, "vdim": a.vdim}
            if a.rot is not None:
                md["rot"] = {"base": a.rot.base, "dims": a.rot.dims}
            if a.q_temp_coef:
                md["q_temp"] = {"coef": a.q_temp_coef, "every": a.q_temp_every}
            if a.softcap:
                md["softcap"] = a.softcap
            return md
        out = []
        for l in self.layers:
            m = l.mixer
            if l.type == "attention":
                md = att(m)
            elif l.type == "parallel":
                md = {"left": att(m.left), "left_scale": m.left_scale, "right_scale": m.right_scale,
                      "right": {"conv": m.right.conv, "dt_rank": m.right.dt_rank, "inner": m.right.inner, "state": m.right.state}}
            else:
                md = {"dim": m.dim, "heads": m.heads, "tau": m.tau, "vdim": m.vdim}
            mlp = None
            if l.mlp is not None:
                mlp = {"expert": {"ff": l.mlp.expert_ff}, "kind": "moe", "router": {"experts": l.mlp.experts, "top": l.mlp.top}}
            out.append({"type": l.type, "mixer": md, "mlp": mlp})
        return {"architecture": "Vefunex", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
                "residual_mult": self.residual_mult, "logit_softcap": self.logit_softcap, "canon": {"taps": self.canon_taps}, "layers": out,
                "kv_page_size": self.kv_page_size, "eos_token_id": self.eos_token_id, "pad_token_id": self.pad_token_id}


# --------------------------------------------------------------------------------------------------------------------- Munevik
@dataclass
class GatedLruSpec:
    """Gated linear recurrent unit: `width` channels with one fp32 state each; an input branch behind a causal convolution of `conv`
    taps (with bias, no activation) whose recurrence and input gates are block-diagonal projections of `blocks` square matrices,
    and a gelu branch that multiplies the states. S <- a S + sqrt(1 - a^2) i u with a = exp(-decay_scale r softplus(lam))."""
    width: int
    blocks: int
    conv: int
    decay_scale: float = 8.0


@dataclass
class ClampedMlpSpec:
    """g = min(W_gate x, limit), u = clamp(W_up x, -limit, limit), W_down (g sigmoid(1.702 g) (u + 1)), no biases."""
    ff: int
    limit: float


@dataclass
class GroupedMoeSpec:
    """`experts` gated silu experts (no biases) of width expert_ff, `top` per token by the largest sigmoid router scores, weights
    score * scale. groups / keep: experts form that many equal groups of neighbours, a group is scored by the sum of its two
    largest scores, and only experts of the best `keep` groups can be chosen (1 / 1: no groups). shared_ff: width of an expert of
    the same form that every token passes and that is added as it is (None: none)."""
    experts: int
    top: int
    expert_ff: int
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    shared_ff: Optional[int] = None


@dataclass
class MunevikLayerSpec:
    type: str                      # 'latent_attention' | 'rglru'
    mixer: object                  # LatentAttentionSpec | GatedLruSpec
    mlp: object                    # ClampedMlpSpec | GroupedMoeSpec | None


@dataclass
class MunevikConfig:
    model_type: str = "munevik"
    vocab_size: int = 0
    hidden_size: int = 0
    norm_eps: float = 1e-6
    postln_alpha: float = 1.0      # a sublayer's residual: x <- norm(postln_alpha * x + sublayer(x))
    layers: List[MunevikLayerSpec] = field(default_factory=list)
    kv_page_size: int = 64         # engine knob: tokens per cache page
    eos_token_id: int = -1
    pad_token_id: int = 0

    MIXERS = ("latent_attention", "rglru")
    SWISH_SLOPE = 1.702            # the dense feed-forward's gate is g * sigmoid(SWISH_SLOPE * g)
    UP_SHIFT = 1.0                 # ... times (u + UP_SHIFT)

    @staticmethod
    def _latent(m: dict, i: int, layers: list) -> LatentAttentionSpec:
        rot, mask, src = m.get("rot") or {}, m.get("mask") or {}, m.get("kv_from")
        rspec = RotarySpec(dims=int(rot.get("dims", m["rot_dim"])), base=float(rot.get("base", 10000.0)))
        spec = LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                                   scale=float(m["scale"]), rot=rspec, window=int(mask["size"]) if mask.get("size") is not None else None,
                                   head_gate=True, kv_from=int(src) if src is not None else None)
        if min(spec.heads, spec.dim, spec.vdim, spec.kv_rank) < 1 or spec.rot_dim < 0 or rspec.dims % 2 or not 0 <= rspec.dims <= spec.rot_dim or \
                (spec.window is not None and spec.window < 1):
            raise ValueError(f"layer {i}: inconsistent attention sizes")
        if spec.kv_from is not None:
            s = layers[spec.kv_from].mixer if 0 <= spec.kv_from < i else None
            if not isinstance(s, LatentAttentionSpec) or s.kv_from is not None:
                raise ValueError(f"layer {i}: kv_from must name an earlier latent-attention layer with a cache of its own")
            if (s.kv_rank, s.rot_dim, s.rot) != (spec.kv_rank, spec.rot_dim, spec.rot):
                raise ValueError(f"layer {i}: kv_rank, rot_dim and rotation must be those of layer {spec.kv_from}")
        return spec

    @classmethod
    def from_dict(cls, d: dict) -> "MunevikConfig":
        layers = []
        for i, ld in enumerate(d["layers"]):
            typ, m = ld["type"], ld["mixer"]
            if typ == "latent_attention":
                mix = cls._latent(m, i, layers)
            elif typ == "rglru":
                mix = GatedLruSpec(width=int(m["width"]), blocks=int(m["blocks"]), conv=int(m["conv"]))
                if min(mix.width, mix.blocks, mix.conv) < 1 or mix.width % mix.blocks:
                    raise ValueError(f"layer {i}: inconsistent recurrence sizes")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {typ!r}")
            md, mlp = ld.get("mlp"), None
            if md:
                kind = md.get("kind", "dense")
                if kind == "dense":
                    mlp = ClampedMlpSpec(ff=int(md["ff"]), limit=float(md["limit"]))
                elif kind == "moe":
                    r, g, sh = md["router"], md["router"].get("groups") or {}, md.get("shared")
                    mlp = GroupedMoeSpec(experts=int(r["experts"]), top=int(r["top"]), expert_ff=int(md["expert"]["ff"]), groups=int(g.get("count", 1)),
                                         keep=int(g.get("keep", g.get("count", 1))), scale=float(r.get("scale", 1.0)),
                                         shared_ff=int(sh["ff"]) if sh else None)
                    if min(mlp.experts, mlp.top, mlp.expert_ff, mlp.groups) < 1 or mlp.experts % mlp.groups or not 1 <= mlp.keep <= mlp.groups:
                        raise ValueError(f"layer {i}: inconsistent expert sizes")
                    if mlp.top > mlp.keep * (mlp.experts // mlp.groups):
                        raise ValueError(f"layer {i}: fewer experts can be chosen than a token uses")
                else:
                    raise ValueError(f"layer {i}: unknown feed-forward kind {kind!r}")
            layers.append(MunevikLayerSpec(type=typ, mixer=mix, mlp=mlp))
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), norm_eps=float((d.get("norm") or {}).get("eps", 1e-6)),
                   postln_alpha=float(d.get("postln_alpha", 1.0)), layers=layers, kv_page_size=int(d.get("kv_page_size", 64)),
                   eos_token_id=int(d.get("eos_token_id", -1)), pad_token_id=int(d.get("pad_token_id", 0)))

    def to_dict(self) -> dict:
        """The config.json form (round-trips through from_dict)."""
        out = []
        for l in self.layers:
            m, s, mlp = l.mixer, l.mlp, None
            if isinstance(m, LatentAttentionSpec):
                md = {"dim": m.dim, "heads": m.heads, "kv_rank": m.kv_rank, "rot": {"base": m.rot.base, "dims": m.rot.dims}, "rot_dim": m.rot_dim,
                      "scale": m.scale, "vdim": m.vdim}
                if m.window is not None:
                    md["mask"] = {"size": m.window}
                if m.kv_from is not None:
                    md["kv_from"] = m.kv_from
            else:
                md = {"blocks": m.blocks, "conv": m.conv, "width": m.width}
            if isinstance(s, ClampedMlpSpec):
                mlp = {"ff": s.ff, "kind": "dense", "limit": s.limit}
            elif isinstance(s, GroupedMoeSpec):
                mlp = {"expert": {"ff": s.expert_ff}, "kind": "moe", "shared": {"ff": s.shared_ff} if s.shared_ff else None,
                       "router": {"experts": s.experts, "groups": {"count": s.groups, "keep": s.keep}, "scale": s.scale, "top": s.top}}
            out.append({"type": l.type, "mixer": md, "mlp": mlp})
        return {"architecture": "Munevik", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
                "postln_alpha": self.postln_alpha, "layers": out, "kv_page_size": self.kv_page_size, "eos_token_id": self.eos_token_id,
                "pad_token_id": self.pad_token_id}


# --------------------------------------------------------------------------------------------------------------------- Sorupel
@dataclass
class ChunkAttentionSpec:
    """Softmax attention with grouped heads over chunks of `chunk` positions counted from the start of the sequence (None: over
    everything earlier): a row sees the earlier rows of its own chunk. Queries and keys are RMS-normed over their whole projection, then
    rotated; the values are the keys as projected (so a value is as wide as a key). Scores are scaled and soft-capped (0: off), the
    denominator holds an additional 1, and every head's output is multiplied by a sigmoid of a projection of the mixer's input."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    rot: RotarySpec
    chunk: Optional[int] = None
    softcap: float = 0.0


@dataclass
class StateSpaceSpec:
    """State-space mixer with one step size per head (Mamba-2): `heads` heads of vdim channels with a fp32 state [state, vdim] each, input
    and output vectors B, C [state] shared by the heads of a group, a causal convolution of `conv` taps (with bias) and silu in front;
    S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x, gated by silu(z), then RMS-normed in norm_groups equal parts."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int = 1

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_channels(self) -> int:
        return self.inner + 2 * self.groups * self.state


@dataclass
class BigramSpec:
    """A second embedding row per token, chosen by (previous * mul_prev + current * mul_cur) mod buckets; a sequence's first token has a
    row of its own behind the buckets."""
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass
class SorupelLayerSpec:
    type: str                      # 'latent_attention' | 'mamba2' | 'attention'
    mixer: object                  # LatentAttentionSpec | StateSpaceSpec | ChunkAttentionSpec
    mlp: Optional[DenseMlpSpec]


@dataclass
class SorupelConfig:
    model_type: str = "sorupel"
    vocab_size: int = 0
    hidden_size: int = 0
    norm_eps: float = 1e-6
    bigram: Optional[BigramSpec] = None
    layers: List[SorupelLayerSpec] = field(default_factory=list)
    kv_page_size: int = 64         # engine knob: tokens per cache page
    eos_token_id: int = -1
    pad_token_id: int = 0

    MIXERS = ("latent_attention", "mamba2", "attention")

    @staticmethod
    def _rotary(m: dict, dims: int, i: int) -> RotarySpec:
        rot = m.get("rot") or {}
        spec = RotarySpec(dims=int(rot.get("dims", dims)), base=float(rot.get("base", 10000.0)), halves=True)
        if spec.dims % 2 or not 0 <= spec.dims <= dims or not spec.base > 0:
            raise ValueError(f"layer {i}: rot.dims must be even and at most {dims}")
        return spec

    @classmethod
    def _latent(cls, m: dict, i: int, layers: list) -> LatentAttentionSpec:
        src = m.get("kv_from")
        spec = LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                                   scale=float(m["scale"]), rot=cls._rotary(m, int(m["rot_dim"]), i), sink=True, out_gate=True,
                                   kv_from=int(src) if src is not None else None)
        if min(spec.heads, spec.dim, spec.vdim, spec.kv_rank) < 1 or spec.rot_dim < 0:
            raise ValueError(f"layer {i}: inconsistent attention sizes")
        if spec.kv_from is not None:
            s = layers[spec.kv_from].mixer if 0 <= spec.kv_from < i else None
            if not isinstance(s, LatentAttentionSpec) or s.kv_from is not None:
                raise ValueError(f"layer {i}: kv_from must name an earlier latent-attention layer with a cache of its own")
            if (s.kv_rank, s.rot_dim, s.rot) != (spec.kv_rank, spec.rot_dim, spec.rot):
                raise ValueError(f"layer {i}: kv_rank, rot_dim and rotation must be those of layer {spec.kv_from}")
        return spec

    @classmethod
    def _attention(cls, m: dict, i: int) -> ChunkAttentionSpec:
        size = (m.get("mask") or {}).get("size")
        spec = ChunkAttentionSpec(heads=int(m["heads"]), kv_heads=int(m.get("kv_heads") or m["heads"]), dim=int(m["dim"]), scale=float(m["scale"]),
                                  rot=cls._rotary(m, int(m["dim"]), i), chunk=int(size) if size is not None else None,
                                  softcap=float(m.get("softcap") or 0.0))
        if min(spec.heads, spec.kv_heads, spec.dim) < 1 or spec.heads % spec.kv_heads or (spec.chunk is not None and spec.chunk < 1) or spec.softcap < 0:
            raise ValueError(f"layer {i}: inconsistent attention sizes")
        if int(m.get("vdim", spec.dim)) != spec.dim:
            raise ValueError(f"layer {i}: the values are the keys, so vdim must equal dim")
        return spec

    @classmethod
    def from_dict(cls, d: dict) -> "SorupelConfig":
        layers = []
        for i, ld in enumerate(d["layers"]):
            typ, m = ld["type"], ld["mixer"]
            if typ == "latent_attention":
                mix = cls._latent(m, i, layers)
            elif typ == "attention":
                mix = cls._attention(m, i)
            elif typ == "mamba2":
                mix = StateSpaceSpec(heads=int(m["heads"]), vdim=int(m["vdim"]), state=int(m["state"]), groups=int(m["groups"]), conv=int(m["conv"]),
                                     norm_groups=int(m.get("norm_groups", 1)))
                if min(mix.heads, mix.vdim, mix.state, mix.groups, mix.conv, mix.norm_groups) < 1 or mix.heads % mix.groups or mix.inner % mix.norm_groups:
                    raise ValueError(f"layer {i}: inconsistent state-space sizes")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {typ!r}")
            md, mlp = ld.get("mlp"), None
            if md:
                if md.get("kind", "dense") != "dense":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {md.get('kind')!r}")
                mlp = DenseMlpSpec(ff=int(md["ff"]), bias=False)
                if mlp.ff < 1:
                    raise ValueError(f"layer {i}: a feed-forward needs a width")
            layers.append(SorupelLayerSpec(type=typ, mixer=mix, mlp=mlp))
        b = (d.get("embedding") or {}).get("bigram")
        bigram = BigramSpec(buckets=int(b["buckets"]), mul_prev=int(b["mul_prev"]), mul_cur=int(b["mul_cur"])) if b else None
        if bigram is not None and bigram.buckets < 1:
            raise ValueError("embedding.bigram needs at least one bucket")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), norm_eps=float((d.get("norm") or {}).get("eps", 1e-6)), bigram=bigram,
                   layers=layers, kv_page_size=int(d.get("kv_page_size", 64)), eos_token_id=int(d.get("eos_token_id", -1)),
                   pad_token_id=int(d.get("pad_token_id", 0)))

    def to_dict(self) -> dict:
        """The config.json form (round-trips through from_dict)."""
        out = []
        for l in self.layers:
            m = l.mixer
            if isinstance(m, StateSpaceSpec):
                md = {"conv": m.conv, "groups": m.groups, "heads": m.heads, "norm_groups": m.norm_groups, "state": m.state, "vdim": m.vdim}
            else:
                md = {"dim": m.dim, "heads": m.heads, "rot": {"base": m.rot.base, "dims": m.rot.dims}, "scale": m.scale}
                if isinstance(m, LatentAttentionSpec):
                    md.update(kv_rank=m.kv_rank, rot_dim=m.rot_dim, vdim=m.vdim)
                    if m.kv_from is not None:
                        md["kv_from"] = m.kv_from
                else:
                    md.update(kv_heads=m.kv_heads, vdim=m.dim)
                    if m.chunk is not None:
                        md["mask"] = {"size": m.chunk}
                    if m.softcap:
                        md["softcap"] = m.softcap
            out.append({"type": l.type, "mixer": md, "mlp": {"ff": l.mlp.ff, "kind": "dense"} if l.mlp is not None else None})
        emb = {}
        if self.bigram is not None:
            emb["bigram"] = {"buckets": self.bigram.buckets, "mul_cur": self.bigram.mul_cur, "mul_prev": self.bigram.mul_prev}
        return {"architecture": "Sorupel", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps}, "embedding": emb,
                "layers": out, "kv_page_size": self.kv_page_size, "eos_token_id": self.eos_token_id, "pad_token_id": self.pad_token_id}
