"""Model shape descriptions for the MLA-family MoE architectures the engine runs.

One dataclass covers the five architecture names of the reference's config schema
(``config/schema.json`` -> ``model.architecture``: deepseek_v3, glm_moe_dsa, kimi_k25,
deepseek_v4, glm5_next) through feature switches: RoPE or NoPE MLA, DSA indexer (with
IndexShare / IndexPool), KDA linear-attention layers and mHC residual streams.  The
presets reproduce the dimensions of the reference's test-data model configs
(``test-data/{DeepSeek-V3.2,GLM-5.2,GLM-5.3-Flash}/config.json``), and
``from_hf_config`` reads the same HuggingFace ``config.json`` files.
Reference: src/model/model_config.h:19-204.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field, asdict
from typing import List, Optional

ARCHITECTURES = ("deepseek_v3", "glm_moe_dsa", "kimi_k25", "deepseek_v4", "glm5_next", "gazutar", "rubasun", "fasodra", "nivasun")

RECURRENT_KINDS = ("channel_delta", "head_delta", "time_mix")


@dataclass
class BlockSpec:
    """One layer of a model that is described layer by layer (``ModelConfig.blocks``): a mixer and an optional feed-forward, dense or a
    mixture of experts, each with sizes of its own."""
    # "attention" | "latent_attention" | "channel_delta" (gated delta rule, a decay per key channel and low-rank gates) | "head_delta" (gated delta
    # rule, a decay per head and a full-rank silu gate) | "time_mix" (token shift, data-dependent decay per key channel, bonus for the current
    # token) | "parallel" (two of the others side by side, see `branches`)
    kind: str = "attention"
    heads: int = 0                    # query heads (attention) / value heads (delta)
    kv_heads: int = 0                 # key-value heads (attention) / query-key heads (delta); divides `heads`
    dim: int = 0                      # query / key head width
    vdim: int = 0                     # value head width
    # attention
    scale: float = 0.0
    window: int = 0                   # sliding window: 0 <= i - j < window (0 = the whole prefix)
    qk_norm: bool = False             # RMS norm over all rows of the q (and of the k) projection
    alibi: bool = False               # linear distance bias, slope 2^(-8 (h + 1) / heads)
    out_gate: bool = False            # heads times sigmoid(W_g h) in front of the output projection
    v_mix: bool = False               # values mixed with those of the first such layer
    chunk: int = 0                    # chunked mask: a position sees the keys of its own chunk (0 = the whole prefix)
    qkv_bias: bool = False            # biases on the q, k and v projections
    head_norm: str = ""               # RMS norm of every q and k head: "" none | "plain" (no weight) | "weight" (one weight for all heads)
    half_rot: int = 0                 # leading channels of q and k heads that are rotated (channel i with i + half_rot / 2), base rot_base
    pair_rot: int = 0                 # the same with adjacent channels (2 i with 2 i + 1)
    shared_kv: bool = False           # no value projection: the values are the keys in front of their rotation
    temp: bool = False                # a learned factor per query head on the scores
    sink: bool = False                # a learned score per head that only the softmax's denominator has
    diff: Optional[float] = None      # differential attention: two maps per head over the same values, rms(o_1 - lambda o_2) (1 - diff) per head with
                                      # lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff
    bias_rows: int = 0                # rows of a learned distance bias table (0: none): one per distance, then logarithmic up to bias_max
    bias_max: int = 0
    # latent attention (one cached row of kv_rank + rot_dim per token for all heads)
    kv_rank: int = 0
    q_rank: int = 0                   # queries through a latent of their own, RMS-normed (0: straight from the input)
    rot_dim: int = 0                  # rotated query / key channels per head, behind `dim` unrotated ones (0: no positions)
    rot_base: float = 10000.0
    kv_from: int = -1                 # layer whose cached rows are attended over (-1: the layer's own)
    head_gate: bool = False           # head h times sigmoid((W_g h)_h)
    # delta rule
    conv: int = 0                     # taps of the short causal convolutions
    decay: str = "softplus"           # log decay: "softplus" -exp(A) softplus(x) | "bounded" decay_bound * sigmoid(exp(A) x)
    decay_bound: float = -5.0
    # two mixers side by side over the same input: "scaled" a * left + b * right (each branch's out_scale), "normed" the mean of both
    # results, each RMS-normed with a weight
    branches: List["BlockSpec"] = field(default_factory=list)
    join: str = "scaled"
    out_scale: float = 1.0
    # feed-forward (dense_ff 0 and experts 0: none)
    dense_ff: int = 0                 # width of a dense gated unit
    experts: int = 0
    identity: int = 0                 # router outputs behind the experts whose "expert" is the input itself
    top: int = 0
    groups: int = 1
    keep: int = 1                     # groups a token may choose from
    ff: int = 0
    # router: scores, selection correction; where a chosen expert's weight goes
    scoring: str = "softmax"          # softmax | sigmoid
    correction: bool = True
    logit_bias: bool = False          # the router's bias is part of the logits: the choice is by them, the weights are their softmax
    unit: str = "glu"                 # the experts' hidden unit: "glu" (gate and up) | "relu2" (square of relu of up, no gate)
    scale_input: bool = False         # the weight multiplies the expert's input instead of its output
    # the experts' gated unit min(g, limit) sigmoid(act_alpha g) (clamp(u, -limit, limit) + act_shift); limit 0: no clamps
    limit: float = 0.0
    act_alpha: float = 1.0
    act_shift: float = 0.0
    shared_ff: int = 0                # an expert for every token (same unit, own limit) times sigmoid of one number per token
    shared_limit: float = 0.0

    def __post_init__(self):
        self.branches = [b if isinstance(b, BlockSpec) else BlockSpec(**b) for b in self.branches]

    @property
    def mixers(self) -> List["BlockSpec"]:
        """The layer's mixers: itself, or the two that run side by side."""
        return self.branches or [self]

    @property
    def recurrent(self) -> bool:
        """The mixer keeps a state per sequence instead of a cache."""
        return self.kind in RECURRENT_KINDS

    @property
    def delta(self) -> bool:
        return self.kind in ("channel_delta", "head_delta")

    @property
    def softmax(self) -> bool:
        return self.kind == "attention"

    @property
    def latent(self) -> bool:
        return self.kind == "latent_attention"

    @property
    def maps(self) -> int:
        """Attention maps of a head."""
        return 2 if self.diff is not None else 1

    @property
    def has_ff(self) -> bool:
        return self.dense_ff > 0 or self.experts > 0


@dataclass
class ModelConfig:
    name: str = "tiny"
    architecture: str = "deepseek_v3"
    hidden: int = 256
    n_layers: int = 4
    vocab: int = 1024
    rms_eps: float = 1e-6
    # MLA
    n_heads: int = 8
    q_lora: int = 128
    kv_lora: int = 64
    qk_nope: int = 32
    qk_rope: int = 16
    v_head: int = 32
    rope_theta: float = 10000.0
    rope_yarn_factor: float = 1.0
    rope_yarn_orig_max: int = 4096
    rope_yarn_beta_fast: float = 32.0
    rope_yarn_beta_slow: float = 1.0
    rope_yarn_mscale_all_dim: float = 0.0
    max_position: int = 8192
    # FFN / MoE
    dense_inter: int = 512
    first_k_dense: int = 1
    n_routed: int = 16
    top_k: int = 4
    n_mtp: int = 0                      # multi-token-prediction blocks after the main stack (layer ids n_layers .. n_layers + n_mtp - 1)
    n_shared: int = 1
    num_hash_layers: int = 0            # MoE layers with index < this route by a token-id table (`moe.tid2eid`, DeepSeek-V4 hash layers) instead of top-k
    moe_inter: int = 128
    scoring: str = "softmax"          # sigmoid | softmax | sqrtsoftplus
    n_group: int = 1
    topk_group: int = 1
    routed_scale: float = 1.0
    norm_topk_prob: bool = True
    router_bias: bool = False         # e_score_correction_bias
    swiglu_limit: float = 0.0
    # DSA indexer (0 heads = dense attention)
    index_n_heads: int = 0
    index_head_dim: int = 128
    index_topk: int = 2048
    index_topk_freq: int = 1          # IndexShare: every freq-th sparse layer recomputes
    index_kpool: int = 1              # IndexPool: tokens per pooled indexer entry
    index_rope_dim: int = 0
    # layer types: "mla" | "kda"
    layer_types: List[str] = field(default_factory=list)
    # KDA
    kda_heads: int = 0
    kda_head_dim: int = 128
    kda_conv: int = 4
    kda_rank: int = 128
    kda_lower_bound: float = -5.0
    # mHC
    hc_mult: int = 1
    hc_eps: float = 1e-6
    hc_sinkhorn_iters: int = 20
    hc_post_mult: float = 2.0
    # weight formats for the synthetic / loaded checkpoint
    expert_quant: str = "bf16"        # bf16 | fp8_e4m3 | nvfp4 | gguf_q4_k ...
    dense_quant: str = "bf16"         # attention / dense FFN / shared expert
    eos_token_ids: List[int] = field(default_factory=list)
    # models described layer by layer (models/block_model.py); empty for the MLA family
    blocks: List[BlockSpec] = field(default_factory=list)
    norm_kind: str = "rms"            # "rms" | "layer" (with bias) | "tanh" (dynamic tanh, element-wise): the norms of the residual stream
    norm_place: str = "post"          # "post": on every sublayer's output | "sandwich": in front of every sublayer and on its output | "pre": in front
                                      # | "parallel": one norm in front of a layer, whose output both sublayers read: x + mixer(h) + ff(h)
    norm_scalar: bool = False         # the norms' weights are one number each
    input_conv: int = 0               # taps of a causal convolution per channel that is added to what a mixer reads (0: none)
    loop: List[int] = field(default_factory=list)      # [start, stop, times]: layers start .. stop - 1 run `times` times in a row, every pass with a cache
                                                       # of its own and a learned vector added to the stream in front of it
    bigram: List[int] = field(default_factory=list)    # [buckets, mul_prev, mul_cur]: a table of buckets + 1 rows, row (prev mul_prev + cur mul_cur) mod
                                                       # buckets added to a token's embedding (the last row: no previous token)
    softcap: float = 0.0              # logits <- softcap tanh(logits / softcap) (0: none)
    streams: int = 0                  # hyper-connections: copies of the residual stream with learned static mixing (0: one plain stream)
    residual_mult: float = 1.0        # factor on every sublayer's output (with `streams`)
    logit_scale: float = 1.0
    embed_scale: float = 1.0
    side_dim: int = 0                 # width of a layer's slice of the per-token side table (0: no such table)

    def __post_init__(self):
        self.blocks = [b if isinstance(b, BlockSpec) else BlockSpec(**b) for b in self.blocks]
        if self.blocks:
            self.n_layers = len(self.blocks)
            self.layer_types = [b.kind for b in self.blocks]
        if not self.layer_types:
            self.layer_types = ["mla"] * self.n_layers
        assert len(self.layer_types) == self.n_layers
        assert self.architecture in ARCHITECTURES
        if self.loop and not (len(self.loop) == 3 and 0 <= self.loop[0] < self.loop[1] <= self.n_layers and self.loop[2] >= 1 and self.blocks):
            raise ValueError(f"layers {self.loop[0]} to {self.loop[1]} of {self.n_layers} cannot run {self.loop[-1]} times")
        for i, b in enumerate(self.blocks):
            if b.maps > 1 and (b.kind != "attention" or b.alibi or b.bias_rows or b.sink or b.out_gate or b.head_gate):
                raise ValueError(f"layer {i}: differential attention comes without distance biases, sinks and gates")
            if b.shared_kv and (b.vdim != b.dim or b.maps > 1 or b.qkv_bias or b.v_mix):
                raise ValueError(f"layer {i}: heads of {b.dim} key channels cannot be values of {b.vdim}")
            if b.branches:
                m = b.mixers
                if b.kind != "parallel" or len(m) != 2 or any(x.branches or x.latent or x.v_mix for x in m) or sum(x.recurrent for x in m) > 1 or sum(x.softmax for x in m) > 1:
                    raise ValueError(f"layer {i}: side by side go two mixers, at most one with a cache and one with a state")
            if b.kv_from >= 0:
                src = self.blocks[b.kv_from] if b.kv_from < i else None
                if src is None or not src.latent or src.kv_from >= 0 or (src.kv_rank, src.rot_dim, src.rot_base) != (b.kv_rank, b.rot_dim, b.rot_base) or self.loop:
                    raise ValueError(f"layer {i}: layer {b.kv_from} has no latent rows of its kind to share")

    # ---- derived ----
    @property
    def qk_head(self) -> int:
        return self.qk_nope + self.qk_rope

    @property
    def has_indexer(self) -> bool:
        return self.index_n_heads > 0

    @property
    def mhc(self) -> bool:
        return self.hc_mult > 1

    def is_moe_layer(self, i: int) -> bool:
        if self.blocks:
            return i < len(self.blocks) and self.blocks[i].experts > 0
        return i >= self.first_k_dense and self.n_routed > 0

    def is_hash_layer(self, i: int) -> bool:
        """The layer's experts come from the token id (table row), not from a top-k over the router scores."""
        return self.is_moe_layer(i) and i < self.num_hash_layers

    def is_kda_layer(self, i: int) -> bool:
        """The layer keeps a recurrent state per sequence: KDA, a recurrent block, or a block with one beside attention."""
        if i < len(self.blocks):
            return any(b.recurrent for b in self.blocks[i].mixers)
        return i < len(self.layer_types) and self.layer_types[i] == "kda"       # multi-token-prediction blocks (i >= n_layers) are MLA layers

    @property
    def keeps_state(self) -> bool:
        """A sequence has state that cannot be rolled back: recurrent layers, or the inputs that convolutions look back at."""
        return self.input_conv > 1 or any(self.is_kda_layer(i) for i in range(self.n_layers))

    def layer_runs(self) -> List[tuple]:
        """[(layer, number of the pass that starts in front of it or -1)] in the order in which the layers run."""
        if not self.loop:
            return [(i, -1) for i in range(self.n_layers)]
        a, b, n = self.loop
        return ([(i, -1) for i in range(a)] + [(i, t if i == a else -1) for t in range(n) for i in range(a, b)] + [(i, -1) for i in range(b, self.n_layers)])

    def mla_layers(self) -> List[int]:
        return [i for i in range(self.n_layers) if not self.is_kda_layer(i)]

    def index_source_layer(self, i: int) -> int:
        """Sparse layer whose indexer selection layer ``i`` uses (IndexShare)."""
        mla = self.mla_layers()
        j = mla.index(i)
        return mla[(j // self.index_topk_freq) * self.index_topk_freq]

    @property
    def softmax_scale(self) -> float:
        s = self.qk_head ** -0.5
        if self.rope_yarn_factor > 1.0 and self.rope_yarn_mscale_all_dim > 0:
            m = 0.1 * self.rope_yarn_mscale_all_dim * math.log(self.rope_yarn_factor) + 1.0
            s *= m * m
        return s

    def rope_inv_freq(self, dim: Optional[int] = None) -> List[float]:
        """Inverse frequencies for ``dim`` rotary dims, with the YaRN correction.
        Reference: src/compute/rope_table.cpp (YaRN ramp between beta_fast and beta_slow)."""
        d = dim if dim is not None else self.qk_rope
        if d <= 0:
            return []
        base = [self.rope_theta ** (-(2.0 * i) / d) for i in range(d // 2)]
        f = self.rope_yarn_factor
        if f <= 1.0:
            return base

        def corr_dim(rot):
            return d * math.log(self.rope_yarn_orig_max / (rot * 2 * math.pi)) / (2 * math.log(self.rope_theta))

        lo = max(math.floor(corr_dim(self.rope_yarn_beta_fast)), 0)
        hi = min(math.ceil(corr_dim(self.rope_yarn_beta_slow)), d - 1)
        if lo == hi:
            hi += 0.001
        out = []
        for i, fr in enumerate(base):
            ramp = min(max((i - lo) / (hi - lo), 0.0), 1.0)
            smooth = 1.0 - ramp
            out.append(fr / f * (1 - smooth) + fr * smooth)
        return out

    # ---- parameter counts (for sizing / autoconfig) ----
    def expert_params(self) -> int:
        return 3 * self.hidden * self.moe_inter

    def n_moe_layers(self) -> int:
        return sum(1 for i in range(self.n_layers) if self.is_moe_layer(i))

    def to_json(self) -> str:
        return json.dumps(asdict(self), indent=1)

    @classmethod
    def from_json(cls, s: str) -> "ModelConfig":
        return cls(**json.loads(s))


def tiny_mla_moe() -> ModelConfig:
    """The CPU-plumbing model: 4 layers (layer 0 dense FFN 512, layers 1-3 MoE), hidden 256,
    8 heads, q_lora 128, kv_lora 64, nope 32, rope 16, v 32, 16 experts top-4 softmax + 1 shared,
    expert FFN 128, vocab 1024."""
    return ModelConfig(name="tiny-mla-moe")


def tiny_glm5_next(n_layers: int = 4) -> ModelConfig:
    """A shrunken glm5_next (KDA + NoPE sparse MLA + mHC + IndexPool) for tests."""
    lt = ["mla" if (i % 4) == 3 else "kda" for i in range(n_layers)]
    return ModelConfig(
        name="tiny-glm5-next", architecture="glm5_next", hidden=256, n_layers=n_layers, vocab=1024, rms_eps=1e-5,
        n_heads=4, q_lora=128, kv_lora=64, qk_nope=64, qk_rope=0, v_head=64, dense_inter=512, first_k_dense=1,
        n_routed=16, top_k=4, n_shared=1, moe_inter=128, scoring="sigmoid", routed_scale=2.5, router_bias=True,
        swiglu_limit=10.0, index_n_heads=4, index_head_dim=128, index_topk=32, index_kpool=4, layer_types=lt,
        kda_heads=2, kda_head_dim=128, kda_rank=32, hc_mult=4)


def tiny_deepseek_v32(n_layers: int = 3) -> ModelConfig:
    """A shrunken DeepSeek-V3.2 shape (RoPE MLA + DSA indexer + grouped sigmoid routing)."""
    return ModelConfig(
        name="tiny-deepseek-v32", architecture="deepseek_v3", hidden=256, n_layers=n_layers, vocab=1024,
        n_heads=8, q_lora=128, kv_lora=64, qk_nope=32, qk_rope=16, v_head=32, dense_inter=512, first_k_dense=1,
        n_routed=32, top_k=4, n_shared=1, moe_inter=128, scoring="sigmoid", n_group=4, topk_group=2,
        routed_scale=2.5, router_bias=True, index_n_heads=4, index_topk=32, index_rope_dim=16,
        rope_yarn_factor=40.0, rope_yarn_mscale_all_dim=1.0)


def deepseek_v3_2() -> ModelConfig:
    return ModelConfig(
        name="DeepSeek-V3.2", architecture="deepseek_v3", hidden=7168, n_layers=61, vocab=129280, rms_eps=1e-6,
        n_heads=128, q_lora=1536, kv_lora=512, qk_nope=128, qk_rope=64, v_head=128, rope_theta=10000.0,
        rope_yarn_factor=40.0, rope_yarn_orig_max=4096, rope_yarn_mscale_all_dim=1.0, max_position=163840,
        dense_inter=18432, first_k_dense=3, n_routed=256, top_k=8, n_shared=1, moe_inter=2048, scoring="sigmoid",
        n_group=8, topk_group=4, routed_scale=2.5, router_bias=True, index_n_heads=64, index_head_dim=128,
        index_topk=2048, index_rope_dim=64, expert_quant="fp8_e4m3", dense_quant="fp8_e4m3", eos_token_ids=[1])


def glm_5_2() -> ModelConfig:
    return ModelConfig(
        name="GLM-5.2", architecture="glm_moe_dsa", hidden=6144, n_layers=78, vocab=154880, rms_eps=1e-5,
        n_heads=64, q_lora=2048, kv_lora=512, qk_nope=192, qk_rope=64, v_head=256, rope_theta=8000000.0,
        max_position=1048576, dense_inter=12288, first_k_dense=3, n_routed=256, top_k=8, n_shared=1, moe_inter=2048,
        scoring="sigmoid", routed_scale=2.5, router_bias=True, index_n_heads=32, index_head_dim=128, index_topk=2048,
        index_topk_freq=4, index_rope_dim=64, expert_quant="gguf_q4_k", dense_quant="bf16",
        eos_token_ids=[154820, 154827, 154829])


def glm_5_3_flash() -> ModelConfig:
    n = 45
    lt = ["mla" if (i % 4) == 3 else "kda" for i in range(n)]
    return ModelConfig(
        name="GLM-5.3-Flash", architecture="glm5_next", hidden=4096, n_layers=n, vocab=154880, rms_eps=1e-5,
        n_heads=64, q_lora=1536, kv_lora=512, qk_nope=256, qk_rope=0, v_head=256, max_position=1048576,
        dense_inter=12288, first_k_dense=3, n_routed=288, top_k=8, n_shared=1, moe_inter=2048, scoring="sigmoid",
        routed_scale=2.5, router_bias=True, swiglu_limit=10.0, index_n_heads=32, index_head_dim=128,
        index_topk=2048, index_kpool=4, layer_types=lt, kda_heads=64, kda_head_dim=128, kda_rank=128,
        kda_lower_bound=-5.0, hc_mult=4, hc_eps=1e-6, hc_sinkhorn_iters=20, expert_quant="nvfp4", dense_quant="bf16",
        eos_token_ids=[154820, 154827, 154829])


def _gazutar(name, width, n_layers, vocab, attn, delta, router, ff, every=3, scale=None) -> ModelConfig:
    """A Gazutar shape: every ``every``-th layer is attention, the others are delta-rule layers."""
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    layers = [{"type": "attention", "mixer": attn, "mlp": mlp} if i % every == every - 1 else {"type": "channel_delta", "mixer": delta, "mlp": mlp}
              for i in range(n_layers)]
    return gazutar_config({"name": name, "layers": layers, "logit_scale": scale or 1.0, "norm": {"eps": 1e-5}, "vocab": vocab, "width": width})


def tiny_gazutar() -> ModelConfig:
    """A small Gazutar shape for tests and smoke runs."""
    return _gazutar("tiny-gazutar", 192, 5, 320, {"heads": 6, "kv_heads": 2, "dim": 32, "vdim": 48, "scale": 0.2, "mask": {"size": 40}, "v_mix": True},
                    {"heads": 4, "kv_heads": 2, "dim": 48, "vdim": 32, "conv": 3},
                    {"experts": 6, "identity": 2, "top": 2, "groups": {"count": 4, "keep": 2}}, 80, every=2, scale=0.5)


def gazutar_flash() -> ModelConfig:
    """A Gazutar shape with layers of a real model's size (the hidden size, KDA heads and expert width of the GLM-5.3-Flash shape)."""
    return _gazutar("gazutar-flash", 4096, 8, 154880, {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 4096}, "v_mix": True},
                    {"heads": 64, "kv_heads": 64, "dim": 128, "vdim": 128, "conv": 4},
                    {"experts": 64, "identity": 8, "top": 8, "groups": {"count": 8, "keep": 4}}, 2048, every=4)


def _rubasun(name, width, vocab, mixer, dense_ff, experts, top, ff, shared, limits, n_layers, share=2, side=0, scale=1.0) -> ModelConfig:
    """A Rubasun shape: a dense first layer, then expert layers of which every ``share``-th makes latent rows that the ones behind it use."""
    layers = []
    for i in range(n_layers):
        m, src = dict(mixer), 1 + (i - 1) // share * share if i else 0
        if src != i:
            m["kv_from"] = src
        mlp = {"kind": "dense", "ff": dense_ff} if i == 0 else {"kind": "moe", "expert": {"ff": ff, "limit": limits[0]}, "router": {"experts": experts, "top": top},
                                                               "shared": {"ff": shared, "limit": limits[1]}}
        layers.append({"type": "latent_attention", "mixer": m, "mlp": mlp})
    return rubasun_config({"name": name, "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": 1e-5}, "embedding": {"scale": scale}, "token_side": {"dim": side}})


def tiny_rubasun() -> ModelConfig:
    """A small Rubasun shape for tests and smoke runs."""
    return _rubasun("tiny-rubasun", 192, 320, {"heads": 6, "dim": 40, "rot_dim": 16, "vdim": 24, "kv_rank": 80, "rot": {"base": 5000.0, "dims": 16}, "scale": 0.15}, 256,
                    6, 2, 80, 72, (3.0, 2.0), 5, side=20, scale=2.0)


def rubasun_flash() -> ModelConfig:
    """A Rubasun shape with layers of a real model's size."""
    return _rubasun("rubasun-flash", 4096, 154880, {"heads": 32, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "rot": {"base": 1e6, "dims": 64}, "scale": 192 ** -0.5},
                    12288, 64, 8, 2048, 2048, (7.0, 7.0), 8, side=256)


def _fasodra(name, width, vocab, heads, kv, dim, chunk, left, time, delta, experts, top, ff, n_layers, streams=2) -> ModelConfig:
    """A Fasodra shape: chunked attention, attention beside time mixing, chunked attention, attention beside a delta rule, in turns."""
    att = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "bias_max": chunk, "mask": {"size": chunk}}
    lft = {"heads": left[0], "kv_heads": left[1], "dim": left[2], "vdim": left[2], "scale": left[2] ** -0.5, "rot": {"base": 1e5, "dims": left[2] // 2}}
    par = {"left": lft, "right": {"heads": time[0], "dim": time[1]}, "left_scale": 0.7, "right_scale": 0.9}
    par2 = {"left": lft, "right": {"heads": delta[0], "kv_heads": delta[1], "dim": delta[2], "vdim": delta[2], "conv": 4}}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    kinds = [("attention", att), ("parallel", par), ("attention", att), ("parallel_2", par2)]
    return fasodra_config({"name": name, "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "residual_mult": 0.8, "streams": streams,
                           "layers": [{"type": kinds[i % 4][0], "mixer": kinds[i % 4][1], "mlp": mlp} for i in range(n_layers)]})


def tiny_fasodra() -> ModelConfig:
    """A small Fasodra shape for tests and smoke runs."""
    return _fasodra("tiny-fasodra", 192, 320, 6, 2, 32, 40, (4, 2, 48), (5, 24), (4, 2, 40), 6, 2, 80, 4, 3)


def fasodra_flash() -> ModelConfig:
    """A Fasodra shape with layers of a real model's size."""
    return _fasodra("fasodra-flash", 4096, 154880, 32, 8, 128, 4096, (32, 8, 128), (64, 64), (32, 32, 128), 64, 8, 3072, 8)


def _nivasun(name, width, vocab, att, lat, diff, moe, n_layers, loop, taps, buckets) -> ModelConfig:
    """A Nivasun shape: attention, latent attention and differential attention in turns."""
    kinds = [("attention", att), ("latent_attention", lat), ("attention_2", diff)]
    return nivasun_config({"name": name, "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "canon": {"taps": taps}, "logit_softcap": 20.0,
                           "embedding": {"scale": width ** 0.5, "bigram": {"buckets": buckets, "mul_cur": 29, "mul_prev": 53}},
                           "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]},
                           "layers": [{"type": kinds[i % 3][0], "mixer": kinds[i % 3][1], "mlp": moe} for i in range(n_layers)]})


def tiny_nivasun() -> ModelConfig:
    """A small Nivasun shape for tests and smoke runs."""
    return _nivasun("tiny-nivasun", 192, 320, {"heads": 4, "kv_heads": 2, "dim": 48, "vdim": 48, "scale": 0.15, "mask": {"size": 37}, "rot": {"base": 1e4, "dims": 32}},
                    {"heads": 6, "dim": 24, "vdim": 40, "kv_rank": 56, "q_rank": 72, "scale": 0.2, "mask": {"size": 50}},
                    {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 40, "scale": 0.25, "diff": 0.4, "mask": {"size": 29}, "rot": {"base": 500.0, "dims": 12}},
                    {"kind": "moe", "expert": {"ff": 80}, "router": {"experts": 6, "top": 2}, "shared": {"ff": 72}}, 4, (1, 3, 2), 4, 509)


def nivasun_flash() -> ModelConfig:
    """A Nivasun shape with layers of a real model's size."""
    return _nivasun("nivasun-flash", 4096, 154880, {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 4096}, "rot": {"base": 1e6, "dims": 128}},
                    {"heads": 32, "dim": 128, "vdim": 128, "kv_rank": 512, "q_rank": 1536, "scale": 128 ** -0.5, "mask": {"size": 4096}},
                    {"heads": 16, "kv_heads": 8, "dim": 128, "vdim": 256, "scale": 128 ** -0.5, "diff": 0.5, "mask": {"size": 4096}, "rot": {"base": 1e6, "dims": 64}},
                    {"kind": "moe", "expert": {"ff": 2048}, "router": {"experts": 64, "top": 8}, "shared": {"ff": 2048}}, 6, (1, 4, 2), 4, 1 << 20)


PRESETS = {
    "tiny-nivasun": tiny_nivasun,
    "nivasun-flash": nivasun_flash,
    "tiny-fasodra": tiny_fasodra,
    "fasodra-flash": fasodra_flash,
    "tiny-rubasun": tiny_rubasun,
    "rubasun-flash": rubasun_flash,
    "tiny-gazutar": tiny_gazutar,
    "gazutar-flash": gazutar_flash,
    "tiny-mla-moe": tiny_mla_moe,
    "tiny-glm5-next": tiny_glm5_next,
    "tiny-deepseek-v32": tiny_deepseek_v32,
    "deepseek-v3.2": deepseek_v3_2,
    "glm-5.2": glm_5_2,
    "glm-5.3-flash": glm_5_3_flash,
}


def get_preset(name: str) -> ModelConfig:
    return PRESETS[name.lower()]()


def gazutar_config(c: dict) -> ModelConfig:
    """Gazutar: post-norm residual stream with layer norms; windowed ALiBi attention with whole-projection query / key norms, value mixing
    and an output gate, or gated delta-rule layers with a decay per key channel; grouped softmax routing with identity experts."""
    blocks = []
    for i, L in enumerate(c["layers"]):
        m = L["mixer"]
        b = BlockSpec(kind=L["type"], heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"])
        if L["type"] == "attention":
            b.scale, b.window, b.v_mix = float(m["scale"]), int((m.get("mask") or {}).get("size", 0)), bool(m.get("v_mix", False))
            b.qk_norm = b.alibi = b.out_gate = True
        elif L["type"] == "channel_delta":
            b.conv = int(m["conv"])
        else:
            raise ValueError(f"layer {i}: unknown mixer type {L['type']!r}")
        mlp = L.get("mlp")
        if mlp:
            if mlp.get("kind", "moe") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            r = mlp["router"]
            g = r.get("groups") or {}
            b.experts, b.top, b.identity, b.ff = int(r["experts"]), int(r["top"]), int(r.get("identity", 0) or 0), int(mlp["expert"]["ff"])
            b.groups, b.keep = int(g.get("count", 1)), int(g.get("keep", 1))
        blocks.append(b)
    moe = [b for b in blocks if b.experts]
    att = [b for b in blocks if not b.recurrent]
    rec = [b for b in blocks if b.recurrent]
    return ModelConfig(
        name=c.get("name", "Gazutar"), architecture="gazutar", hidden=c["width"], vocab=c["vocab"], rms_eps=float(c["norm"]["eps"]), norm_kind="layer",
        logit_scale=float(c.get("logit_scale", 1.0)), blocks=blocks, n_heads=max((b.heads for b in att), default=1), q_lora=0, kv_lora=0, qk_nope=0, qk_rope=0,
        v_head=max((b.vdim for b in att), default=0), dense_inter=0, first_k_dense=0, n_routed=max((b.experts for b in moe), default=0),
        top_k=max((b.top for b in moe), default=0), n_shared=0, moe_inter=max((b.ff for b in moe), default=0), norm_topk_prob=False, router_bias=True,
        kda_heads=max((b.heads for b in rec), default=0), kda_head_dim=max((b.dim for b in rec), default=0), max_position=int(c.get("max_position", 1 << 20)))


def rubasun_config(c: dict) -> ModelConfig:
    """Rubasun: dynamic-tanh norms around every sublayer; latent attention with rotary positions, a gate per head and cached rows that later layers
    may share; dense or expert feed-forwards (sigmoid scores on the experts' inputs, clamped and shifted gated units, a gated shared expert); a
    table of per-token inputs for every layer."""
    blocks = []
    for i, L in enumerate(c["layers"]):
        if L["type"] != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer type {L['type']!r}")
        m, src = L["mixer"], L["mixer"].get("kv_from")
        rot = m.get("rot") or {}
        if int(rot.get("dims", m["rot_dim"])) != m["rot_dim"]:
            raise ValueError(f"layer {i}: {rot['dims']} rotary channels in a rotated part of {m['rot_dim']}")
        b = BlockSpec(kind=L["type"], heads=m["heads"], kv_heads=1, dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]), kv_rank=m["kv_rank"], rot_dim=m["rot_dim"],
                      rot_base=float(rot.get("base", 10000.0)), kv_from=-1 if src is None else int(src), head_gate=True)
        mlp = L.get("mlp")
        if mlp and mlp["kind"] == "dense":
            b.dense_ff = int(mlp["ff"])
        elif mlp and mlp["kind"] == "moe":
            sh = mlp.get("shared") or {}
            b.experts, b.top, b.ff, b.limit = int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"]), float(mlp["expert"]["limit"])
            b.scoring, b.correction, b.scale_input, b.act_alpha, b.act_shift = "sigmoid", False, True, 1.702, 1.0
            b.shared_ff, b.shared_limit = int(sh.get("ff", 0)), float(sh.get("limit", 0.0))
        elif mlp:
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        blocks.append(b)
    moe = [b for b in blocks if b.experts]
    top = lambda key, of=blocks: max((getattr(b, key) for b in of), default=0)
    return ModelConfig(
        name=c.get("name", "Rubasun"), architecture="rubasun", hidden=c["width"], vocab=c["vocab"], rms_eps=float(c["norm"]["eps"]), norm_kind="tanh",
        norm_place="sandwich", embed_scale=float((c.get("embedding") or {}).get("scale", 1.0)), side_dim=int((c.get("token_side") or {}).get("dim", 0)),
        blocks=blocks, n_heads=max(1, top("heads")), q_lora=0, kv_lora=top("kv_rank"), qk_nope=top("dim"), qk_rope=top("rot_dim"), v_head=top("vdim"),
        rope_theta=blocks[0].rot_base if blocks else 10000.0, dense_inter=top("dense_ff"), first_k_dense=0, n_routed=top("experts", moe), top_k=top("top", moe),
        n_shared=0, moe_inter=top("ff", moe), scoring="sigmoid", norm_topk_prob=False, max_position=int(c.get("max_position", 1 << 20)))


def fasodra_config(c: dict) -> ModelConfig:
    """Fasodra: layer norms in front of every sublayer, hyper-connections with static mixing; chunked attention with a learned distance bias, rotary
    attention beside time mixing (a constant factor on each) or beside a delta rule (each result normed), and ungated squared-relu experts."""
    def attention(m, **kw):
        rot = m.get("rot") or {}
        if int(rot.get("dims", 0)) % 2 or int(rot.get("dims", 0)) > m["dim"]:
            raise ValueError(f"{rot['dims']} rotary channels in heads of {m['dim']}")
        return BlockSpec(kind="attention", heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]), qkv_bias=True,
                         half_rot=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)), **kw)

    blocks = []
    for i, L in enumerate(c["layers"]):
        m = L["mixer"]
        if L["type"] == "attention":
            b = attention(m, head_norm="plain", chunk=int((m.get("mask") or {}).get("size", 0)), bias_rows=32, bias_max=int(m["bias_max"]))
        elif L["type"] == "parallel":
            r = m["right"]
            b = BlockSpec(kind="parallel", join="scaled", branches=[
                attention(m["left"], head_gate=True, out_scale=float(m["left_scale"])),
                BlockSpec(kind="time_mix", heads=r["heads"], kv_heads=r["heads"], dim=r["dim"], vdim=r["dim"], out_scale=float(m["right_scale"]))])
        elif L["type"] == "parallel_2":
            r = m["right"]
            b = BlockSpec(kind="parallel", join="normed", branches=[
                attention(m["left"], head_norm="weight"),
                BlockSpec(kind="head_delta", heads=r["heads"], kv_heads=r["kv_heads"], dim=r["dim"], vdim=r["vdim"], conv=int(r["conv"]))])
        else:
            raise ValueError(f"layer {i}: unknown mixer type {L['type']!r}")
        mlp = L.get("mlp")
        if mlp:
            if mlp.get("kind", "moe") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            b.experts, b.top, b.ff = int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"])
            b.correction, b.unit = False, "relu2"
        blocks.append(b)
    moe = [b for b in blocks if b.experts]
    att = [x for b in blocks for x in b.mixers if not x.recurrent]
    rec = [x for b in blocks for x in b.mixers if x.recurrent]
    top = lambda key, of, least=0: max((getattr(b, key) for b in of), default=least)
    return ModelConfig(
        name=c.get("name", "Fasodra"), architecture="fasodra", hidden=c["width"], vocab=c["vocab"], rms_eps=float(c["norm"]["eps"]), norm_kind="layer",
        norm_place="pre", streams=int(c.get("streams") or 1), residual_mult=float(c.get("residual_mult", 1.0)), blocks=blocks, n_heads=max(1, top("heads", att)),
        q_lora=0, kv_lora=0, qk_nope=0, qk_rope=0, v_head=top("vdim", att), dense_inter=0, first_k_dense=0, n_routed=top("experts", moe), top_k=top("top", moe),
        n_shared=0, moe_inter=top("ff", moe), norm_topk_prob=True, kda_heads=top("heads", rec), kda_head_dim=top("dim", rec),
        max_position=int(c.get("max_position", 1 << 20)))


def nivasun_config(c: dict) -> ModelConfig:
    """Nivasun: one norm (with a single weight) in front of a layer whose mixer, behind a short convolution of its input, and experts run side by side; windowed
    attention with shared keys and values, temperatures and sinks, latent attention without positions, differential attention; layers that run several
    times; a bigram embedding; soft-capped logits."""
    blocks = []
    for i, L in enumerate(c["layers"]):
        m = L["mixer"]
        rot = m.get("rot") or {}
        dims, base = int(rot.get("dims", 0)), float(rot.get("base", 10000.0))
        if dims % 2 or dims > m["dim"]:
            raise ValueError(f"layer {i}: {dims} rotary channels in heads of {m['dim']}")
        b = BlockSpec(kind="attention", heads=m["heads"], kv_heads=m.get("kv_heads", 1), dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                      window=int((m.get("mask") or {}).get("size", 0)), rot_base=base)
        if L["type"] == "attention":
            b.half_rot, b.shared_kv, b.temp, b.sink = dims, True, True, True
        elif L["type"] == "latent_attention":
            b.kind, b.kv_rank, b.q_rank, b.out_gate = "latent_attention", int(m["kv_rank"]), int(m["q_rank"]), True
        elif L["type"] == "attention_2":
            b.pair_rot, b.diff = dims, float(m["diff"])
        else:
            raise ValueError(f"layer {i}: unknown mixer type {L['type']!r}")
        mlp = L.get("mlp")
        if mlp:
            if mlp.get("kind", "moe") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            b.experts, b.top, b.ff = int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"])
            b.correction, b.logit_bias, b.shared_ff = False, True, int((mlp.get("shared") or {}).get("ff", 0))
        blocks.append(b)
    emb, loop = c.get("embedding") or {}, c.get("loop")
    bg = emb.get("bigram")
    moe = [b for b in blocks if b.experts]
    top = lambda key, of=blocks, least=0: max((getattr(b, key) for b in of), default=least)
    return ModelConfig(
        name=c.get("name", "Nivasun"), architecture="nivasun", hidden=c["width"], vocab=c["vocab"], rms_eps=float(c["norm"]["eps"]), norm_kind="rms", norm_place="parallel",
        norm_scalar=True, input_conv=int((c.get("canon") or {}).get("taps", 0)), embed_scale=float(emb.get("scale", 1.0)),
        bigram=[int(bg["buckets"]), int(bg["mul_prev"]), int(bg["mul_cur"])] if bg else [], loop=[int(loop["start"]), int(loop["stop"]), int(loop["times"])] if loop else [],
        softcap=float(c.get("logit_softcap") or 0.0), blocks=blocks, n_heads=max(1, top("heads")), q_lora=top("q_rank"), kv_lora=top("kv_rank"), qk_nope=top("dim"), qk_rope=0,
        v_head=top("vdim"), dense_inter=0, first_k_dense=0, n_routed=top("experts", moe), top_k=top("top", moe), n_shared=0, moe_inter=top("ff", moe),
        norm_topk_prob=True, max_position=int(c.get("max_position", 1 << 20)))


# architectures whose config.json is described by its own keys ("architecture": name) rather than HuggingFace ones
NATIVE_CONFIGS = {"gazutar": gazutar_config, "rubasun": rubasun_config, "fasodra": fasodra_config, "nivasun": nivasun_config}


def from_hf_config(path_or_dict) -> ModelConfig:
    """Build a ModelConfig from a ``config.json`` (path or dict): HuggingFace keys, or the keys of a natively described architecture."""
    c = json.load(open(path_or_dict)) if isinstance(path_or_dict, str) else dict(path_or_dict)
    native = NATIVE_CONFIGS.get(str(c.get("architecture", "")).lower())
    if native is not None:
        return native(c)
    c = c.get("text_config", c)
    mt = c.get("model_type", "")
    arch = {"deepseek_v3": "deepseek_v3", "deepseek_v32": "deepseek_v3", "glm_moe_dsa": "glm_moe_dsa",
            "glm5_next_text": "glm5_next", "glm5_next": "glm5_next", "kimi_k25": "kimi_k25",
            "deepseek_v4": "deepseek_v4"}.get(mt, "deepseek_v3")
    n = c["num_hidden_layers"]
    lt_raw = c.get("layer_types")
    lt = ["kda" if t == "linear_attention" else "mla" for t in lt_raw] if lt_raw else ["mla"] * n
    rs = c.get("rope_scaling") or {}
    rp = c.get("rope_parameters") or {}
    la = c.get("linear_attn_config") or {}
    return ModelConfig(
        name=mt or "hf", architecture=arch, hidden=c["hidden_size"], n_layers=n, vocab=c["vocab_size"],
        rms_eps=c.get("rms_norm_eps", 1e-6), n_heads=c["num_attention_heads"], q_lora=c.get("q_lora_rank") or 0,
        kv_lora=c["kv_lora_rank"], qk_nope=c["qk_nope_head_dim"], qk_rope=c.get("qk_rope_head_dim", 0),
        v_head=c["v_head_dim"], rope_theta=float(rp.get("rope_theta", c.get("rope_theta", 10000.0))),
        rope_yarn_factor=float(rs.get("factor", 1.0)), rope_yarn_orig_max=int(rs.get("original_max_position_embeddings", 4096)),
        rope_yarn_beta_fast=float(rs.get("beta_fast", 32)), rope_yarn_beta_slow=float(rs.get("beta_slow", 1)),
        rope_yarn_mscale_all_dim=float(rs.get("mscale_all_dim", 0.0)), max_position=c.get("max_position_embeddings", 8192),
        dense_inter=c["intermediate_size"], first_k_dense=c.get("first_k_dense_replace", 0),
        n_routed=c.get("n_routed_experts", 0), top_k=c.get("num_experts_per_tok", 0), n_shared=c.get("n_shared_experts", 0),
        n_mtp=int(c.get("num_nextn_predict_layers", 0) or 0), num_hash_layers=int(c.get("num_hash_layers", 0) or 0),
        moe_inter=c.get("moe_intermediate_size", 0), scoring=c.get("scoring_func", "softmax"), n_group=c.get("n_group", 1),
        topk_group=c.get("topk_group", 1), routed_scale=c.get("routed_scaling_factor", 1.0),
        norm_topk_prob=c.get("norm_topk_prob", True), router_bias=c.get("topk_method") == "noaux_tc",
        swiglu_limit=float(c.get("swiglu_limit", 0.0) or 0.0), index_n_heads=c.get("index_n_heads", 0),
        index_head_dim=c.get("index_head_dim", 128), index_topk=c.get("index_topk", 2048),
        index_topk_freq=c.get("index_topk_freq", 1) or 1, index_kpool=c.get("index_kpool", 1) or 1,
        index_rope_dim=c.get("qk_rope_head_dim", 0), layer_types=lt, kda_heads=la.get("num_heads", 0),
        kda_head_dim=la.get("head_dim", 128), kda_conv=la.get("short_conv_kernel_size", 4),
        kda_rank=la.get("gate_low_rank", la.get("head_dim", 128)), kda_lower_bound=la.get("gate_lower_bound", -5.0), hc_mult=c.get("hc_mult", 1) if c.get("mhc") else 1,
        hc_eps=c.get("hc_eps", 1e-6), hc_sinkhorn_iters=c.get("hc_sinkhorn_iters", 20),
        eos_token_ids=(c["eos_token_id"] if isinstance(c.get("eos_token_id"), list) else [c.get("eos_token_id", 0)]))
