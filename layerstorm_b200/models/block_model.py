"""Models described layer by layer (``ModelConfig.blocks``) on the device: every layer is a mixer (grouped-query attention, latent attention, a
gated delta rule, time mixing, or two of them side by side) and an optional feed-forward (a dense gated unit or routed experts), each with its own
sizes, around an fp32 residual stream.  The norms stand on every sublayer's output (``norm_place`` "post"), in front of it ("pre") or on both its
sides ("sandwich"; n_in is the identity for "post", n_out for "pre"):

    x <- x + n_out(mixer(n_in(x))),    x <- x + n_out(ffn(n_in(x))),    logits = head(norm(x)) * logit_scale,

and a layer may end with an update from its slice e of a per-token table: x <- x + rms(W_p (gelu(W_g x) * e)).  With ``streams`` there are n copies of
the stream and every sublayer reads and updates them through learned static weights (in, out, mix):

    u = sum_s in_s x_s,    y = residual_mult * f(n_in(u)),    x_t <- sum_s mix_st x_s + out_t y,    logits = head(norm(sum_t x_t)).

With ``norm_place`` "parallel" both sublayers of a layer read one norm and their projections back are one product: x <- x + mixer(h + conv(h)) + ffn(h),
h = n_in(x), where conv is a short causal convolution per channel (``input_conv``; any placement of the norms may have it).  A range of layers may run
several times (``loop``): same weights, a cache and state per pass, a learned vector on the stream in front of each.

Same engine, caches and step protocol as :class:`DeviceModel`: attention layers keep a paged cache (one row of all heads' keys and values per
token; latent layers one row for all heads, which later layers may read instead of keeping their own), recurrent layers an fp32 state per sequence
slot with the convolutions' history (delta rule) or the previous token's input (time mixing); layers with two mixers side by side have both, and
input convolutions the inputs they look back at.  Caches and states are numbered by layer run.  Steps are any mixture of prompt portions and single tokens.

Two precisions.  ``bfloat16``: weights, activations and the cache in bf16, products accumulated in fp32; the residual stream, norms, routing,
attention scores and weights, rotations and the whole recurrence in fp32.  ``float32``: everything in fp32 (FMA units, no reduced-precision
products).

Sizes are padded where kernels want it: the residual width to a multiple of 8, projection blocks to multiples of 8 rows, head widths and
expert widths to the kernels' tiles; padding holds zeros and never reaches a result.
"""
from __future__ import annotations

import logging
import math
from typing import Dict, List, Optional

import torch

from ..ops import _native as nat
from .config import BlockSpec, ModelConfig
from .device_model import ExpertArena, ModelBase, MoeBuffers, QLinear, StepBuffers, TcScratch, _align, expert_layout

FEW_ROWS = 8            # rows per sequence up to which a delta-rule layer runs as one kernel
LONG_ROWS = 64          # rows of a sequence from which its recurrence runs chunk-parallel
EXPAND_ROWS = 128       # rows of a step of one sequence from which latent layers write keys and values out per head ...
EXPAND_BYTES = 1 << 30  # ... while those of all its positions fit this much scratch
NORM_KIND = {"rms": 0, "layer": 1, "tanh": 2}        # as the kernels number them; 3: none
NO_NORM = (3, None, None, None)
SCORING = {"sigmoid": 0, "softmax": 1}
LOGIT_SCORES = 3        # the router's bias is part of the logits
HEAD_NORM = {"": 0, "plain": 1, "weight": 2}


def _sides(b: BlockSpec) -> list:
    """[(name part, mixer)] of a layer: one mixer, or two side by side."""
    return list(zip(("left.", "right."), b.branches)) if b.branches else [("", b)]


def _mixer_shapes(out: dict, p: str, b: BlockSpec, H: int, ranks: tuple):
    """Adds the tensors of a mixer, named behind ``p``."""
    if b.delta:
        k, kw, vw = p + "kda.", b.kv_heads * b.dim, b.heads * b.vdim
        ra, rg = ranks
        out.update({k + "q": (kw, H), k + "k": (kw, H), k + "v": (vw, H), k + "beta": (b.heads, H), k + "conv_q": (kw, b.conv), k + "conv_k": (kw, b.conv),
                    k + "conv_v": (vw, b.conv), k + "a_log": (b.heads,), k + "o_norm": (b.vdim,), k + "o": (H, vw)})
        if b.kind == "head_delta":
            out.update({k + "a": (b.heads, H), k + "g": (vw, H), k + "dt_bias": (b.heads,)})
        else:
            out.update({k + "f_a": (ra, H), k + "g_a": (rg, H), k + "f_b": (b.heads * b.dim, ra), k + "g_b": (vw, rg), k + "dt_bias": (b.heads * b.dim,)})
    elif b.kind == "time_mix":
        k, kw, vw = p + "tmix.", b.heads * b.dim, b.heads * b.vdim
        out.update({k + "r": (kw, H), k + "k": (kw, H), k + "v": (vw, H), k + "g": (vw, H), k + "w1": (ranks[0], H), k + "w2": (kw, ranks[0]), k + "w0": (kw,),
                    k + "u": (b.heads, b.dim), k + "o_norm": (vw,), k + "o": (H, vw)} | {k + "mu_" + n: (H,) for n in "rkvgw"})
    elif b.latent:
        a = p + "attn."
        qw = b.heads * (b.dim + b.rot_dim)
        out.update({a + "q_a": (b.q_rank, H), a + "q_a_norm": (b.q_rank,), a + "q_b": (qw, b.q_rank)} if b.q_rank else {a + "q": (qw, H)})
        out.update({a + "k_b": (b.heads * b.dim, b.kv_rank), a + "v_b": (b.heads * b.vdim, b.kv_rank),
                    a + "o": (H, b.heads * b.vdim)})
        if b.kv_from < 0:
            out.update({a + "kv_a": (b.kv_rank + b.rot_dim, H), a + "kv_a_norm": (b.kv_rank,)})
        if b.out_gate or b.head_gate:
            out[a + "g"] = (b.heads * (b.vdim if b.out_gate else 1), H)
    else:
        a, qw, kw, vw = p + "attn.", b.heads * b.maps * b.dim, b.kv_heads * b.maps * b.dim, b.kv_heads * b.vdim
        out.update({a + "q": (qw, H), a + "k": (kw, H), a + "o": (H, b.heads * b.vdim)} | ({} if b.shared_kv else {a + "v": (vw, H)}))
        out.update({a + n: (b.heads,) for n, has in (("temp", b.temp), ("sink", b.sink)) if has} | ({a + n: (b.dim,) for n in ("lq1", "lk1", "lq2", "lk2")} if b.maps > 1 else {}))
        if b.qkv_bias:
            out.update({a + "q_bias": (qw,), a + "k_bias": (kw,), a + "v_bias": (vw,)})
        if b.qk_norm:
            out.update({a + "q_norm": (qw,), a + "k_norm": (kw,)})
        if b.head_norm == "weight":
            out.update({a + "q_norm": (b.dim,), a + "k_norm": (b.dim,)})
        if b.bias_rows:
            out[a + "rel"] = (b.bias_rows, b.heads)
        if b.out_gate or b.head_gate:
            out[a + "g"] = (b.heads * (b.vdim if b.out_gate else 1), H)
        if b.v_mix:
            out[a + "v_mix"] = ()


def distance_buckets(rows: int, reach: int) -> List[int]:
    """Rows of a learned distance bias table for distances 0 .. reach (further ones: the last): one each up to half the rows, then logarithmic,
    half + floor(log(n / half) / log(reach / half) * (rows - half)).  In integers, so that distances on a border fall where the formula says."""
    half = rows // 2
    if half < 1 or reach <= half:
        raise ValueError(f"a distance bias of {rows} rows up to distance {reach}")
    m, out, k = rows - half, list(range(half)), 0
    for n in range(half, reach + 1):
        while k < m - 1 and n ** m * half ** (k + 1) >= reach ** (k + 1) * half ** m:
            k += 1
        out.append(half + k)
    return out


def block_weight_shapes(cfg: ModelConfig, ranks: Optional[Dict[int, tuple]] = None) -> Dict[str, tuple]:
    """Canonical tensor names and shapes.  ``ranks``: {layer: (decay rank, gate rank)} of delta-rule layers (default: the key head width)."""
    H, out = cfg.hidden, {}
    extra = {"rms": (), "layer": ("bias",), "tanh": ("bias", "alpha")}[cfg.norm_kind]
    norm = lambda p: out.update({p + ".weight": () if cfg.norm_scalar else (H,)} | {f"{p}.{k}": () if k == "alpha" else (H,) for k in extra})
    out["embed.weight"] = out["head.weight"] = (cfg.vocab, H)
    if cfg.side_dim:
        out["side_embed.weight"] = (cfg.vocab, cfg.n_layers * cfg.side_dim)
    if cfg.bigram:
        out["bigram.weight"] = (cfg.bigram[0] + 1, H)
    if cfg.loop:
        out["loop_step"] = (cfg.loop[2], H)
    norm("final_norm")
    for i, b in enumerate(cfg.blocks):
        p = f"layers.{i}."
        if cfg.input_conv:
            out[p + "input_conv"] = (H, cfg.input_conv)
        norm(p + "mix_norm")
        if cfg.norm_place == "sandwich":
            norm(p + "mix_post_norm")
        for side, m in _sides(b):
            _mixer_shapes(out, p + side, m, H, (ranks or {}).get(i, (m.dim, m.dim)))
            if b.branches and b.join == "normed":
                out[p + side + "out_norm"] = (H,)
        if cfg.streams:
            for q in ["mix_hc"] + (["ffn_hc"] if b.has_ff else []):
                out.update({f"{p}{q}.in": (cfg.streams,), f"{p}{q}.out": (cfg.streams,), f"{p}{q}.mix": (cfg.streams, cfg.streams)})
        if b.has_ff and cfg.norm_place != "parallel":
            norm(p + "ffn_norm")
            if cfg.norm_place == "sandwich":
                norm(p + "ffn_post_norm")
        glu = lambda m, ff: out.update({m + "gate": (ff, H), m + "up": (ff, H), m + "down": (H, ff)})
        if b.dense_ff:
            glu(p + "mlp.", b.dense_ff)
        if b.experts:
            m = p + "moe."
            out[m + "router"] = (b.experts + b.identity, H)
            if b.correction or b.logit_bias:
                out[m + "router_bias"] = (b.experts + b.identity,)
            for e in range(b.experts):
                glu(m + f"experts.{e}.", b.ff)
                if b.unit != "glu":
                    del out[m + f"experts.{e}.gate"]
            if b.shared_ff:
                glu(m + "shared.0.", b.shared_ff)
                out[m + "shared_gate"] = (1, H)
        if cfg.side_dim:
            out.update({p + "side.gate": (cfg.side_dim, H), p + "side.proj": (H, cfg.side_dim), p + "side.norm": (H,)})
    return out


def random_block_tensor(name: str, shape: tuple, gen: torch.Generator, device="cpu") -> torch.Tensor:
    """One random tensor with a spread that keeps every mechanism of the design visible."""
    t = torch.empty(shape, dtype=torch.float32, device=device)
    leaf = name.rsplit(".", 1)[-1]
    if leaf.endswith("norm") or name.endswith("norm.weight"):
        return t.normal_(1.0, 0.1, generator=gen)
    if leaf == "a_log":
        return t.uniform_(-3.0, 0.5, generator=gen)
    if leaf == "dt_bias":
        return t.uniform_(-3.0, -1.0, generator=gen)
    if leaf.startswith("conv_") or leaf == "input_conv":
        return t.uniform_(-0.7, 0.7, generator=gen)
    if leaf == "temp":
        return t.uniform_(0.5, 1.5, generator=gen)
    if leaf in ("sink", "loop_step"):
        return t.normal_(0.0, 0.5, generator=gen)
    if leaf in ("lq1", "lk1", "lq2", "lk2"):
        return t.normal_(0.0, 0.1, generator=gen)
    if leaf.startswith("mu_"):
        return t.uniform_(0.1, 0.9, generator=gen)
    if leaf == "w0":
        return t.uniform_(-5.0, 0.5, generator=gen)
    if leaf in ("in", "out") and len(shape) == 1:
        return t.uniform_(0.6, 1.2, generator=gen)
    if leaf == "mix" and "_hc" in name:
        return t.normal_(0.0, 0.15, generator=gen).add_(torch.eye(shape[0], device=device))
    if leaf in ("rel", "u"):
        return t.normal_(0.0, 0.5, generator=gen)
    if leaf == "v_mix":
        return t.uniform_(0.2, 0.6, generator=gen)
    if leaf in ("bias", "router_bias", "q_bias", "k_bias", "v_bias"):
        return t.normal_(0.0, 0.1, generator=gen)
    if leaf == "alpha":
        return t.uniform_(0.4, 1.0, generator=gen)
    if leaf == "weight":                                     # token tables, head
        return t.normal_(0.0, 1.0 if "embed" in name or "bigram" in name else 0.5 / shape[1] ** 0.5, generator=gen)
    return t.normal_(0.0, 1.0 / shape[1] ** 0.5, generator=gen)


class RandomBlockWeights:
    """Canonical state dict of random tensors, made when asked for (a full-size model never exists as a whole in fp32)."""

    def __init__(self, cfg: ModelConfig, seed: int = 0, device="cpu", ranks=None):
        self.shapes, self.device = block_weight_shapes(cfg, ranks), device
        self.gen = torch.Generator(device=device).manual_seed(seed)

    def __contains__(self, name):
        return name in self.shapes

    def __getitem__(self, name):
        return random_block_tensor(name, self.shapes[name], self.gen, self.device)


class BlockWorkspace(StepBuffers):
    """Activation buffers of a step of up to ``R`` rows."""

    def __init__(self, m: "BlockModel", R: int, n_logit_rows: int, max_ctx: int):
        super().__init__(m, R, n_logit_rows)
        z, act, Hp = self.z, m.act_dtype, m.Hp
        # the residual stream in the activation type, what every sublayer reads; with input convolutions what the mixers read stands in front of it
        self.x_pair = z(2, R, Hp, dtype=act) if m.cfg.input_conv else None
        self.x = z(R, Hp, dtype=act) if self.x_pair is None else self.x_pair[1]
        self.x_mix = self.x if self.x_pair is None else self.x_pair[0]
        self.resid = z(R, Hp)
        self.sub = z(R, Hp)
        self.xh = z(n_logit_rows, Hp, dtype=act)
        self.proj = z(R, m.max_proj)
        self.mix = z(R, m.max_mix, dtype=act)        # a mixer's output in front of its output projection
        lat = [b for b in m.cfg.blocks if b.latent]
        att = [(i, b) for i, L in enumerate(m.cfg.blocks) for b in L.mixers if b.softmax]
        self.streams = z(R, m.cfg.streams, Hp) if m.cfg.streams else None
        self.sub2 = z(R, Hp) if any(b.join == "normed" and b.branches for b in m.cfg.blocks) else None
        self.xs = z(5, R, Hp, dtype=act) if any(b.kind == "time_mix" for L in m.cfg.blocks for b in L.mixers) else None      # token-shifted inputs
        if any(b.q_rank for b in lat):
            self.q_low = z(R * max(_align(b.q_rank, 8) for b in lat), dtype=act)
            self.q_up = z(R * max(_align(b.heads * (b.dim + b.rot_dim), 8) for b in lat if b.q_rank))
        if lat:
            self.q_lat = z(R * max(b.heads * m.latent_row(b) for b in lat), dtype=act)
            self.q_nope = z(R * max(b.heads * _align(b.dim, 8) for b in lat), dtype=torch.bfloat16) if not m.f32 and R >= 8 else None
            self.o_lat = z(R * max(b.heads * m.latent_pad(b.kv_rank) for b in lat), dtype=act)
            self.lat_splits = {i: 1 if R > 64 else int(nat.call("lsb_latent_splits", R, b.heads, b.kv_rank, b.rot_dim, min(b.window or max_ctx, max_ctx), int(m.f32)))
                               for i, b in enumerate(m.cfg.blocks) if b.latent}
            self.lat_parts = {i: int(nat.call("lsb_latent_partials", n)) for i, n in self.lat_splits.items()}
            ns = [(b.heads * self.lat_parts[i], m.latent_pad(b.kv_rank)) for i, b in enumerate(m.cfg.blocks) if self.lat_parts.get(i, 1) > 1]
            self.lat_o_part = z(R * max((n * w for n, w in ns), default=1))
            self.lat_ml_part = z(2 * R * max((n for n, _ in ns), default=1))
        dense = max((_align(max(b.dense_ff, b.shared_ff), 8) for b in m.cfg.blocks), default=0)
        self.glu = z(R * dense, dtype=act) if dense and m.cfg.norm_place != "parallel" else None
        self.side = z(R, _align(m.cfg.side_dim, 8), dtype=act) if m.cfg.side_dim else None
        if att:
            self.q = z(R * max(b.heads * b.maps * m.head_pad(b.dim) for _, b in att), dtype=act)
            self.v_first = z(R, max([b.kv_heads * b.vdim for _, b in att if b.v_mix], default=1))
            # key splits of the few-row attention: about two blocks per SM, no split shorter than 64 visible keys
            self.splits = {}
            for i, b in att:
                seen = min(b.window or max_ctx, b.chunk or max_ctx, max_ctx)
                blocks = R * int(nat.call("lsb_attn_blocks", b.heads * b.maps, b.kv_heads * b.maps, b.maps, m.head_pad(b.dim), m.head_pad(b.vdim)))
                self.splits[i] = 1 if (m.f32 or R > 64) else max(1, min(32, 296 // blocks, (seen + 63) // 64))
            ns = [(b.heads * b.maps * self.splits[i], m.head_pad(b.vdim)) for i, b in att if self.splits[i] * b.maps > 1]
            self.o_part = z(R * max((n * w for n, w in ns), default=1))
            self.ml_part = z(2 * R * max((n for n, _ in ns), default=1))
        self.moe: Dict[tuple, MoeBuffers] = {}
        for i, b in enumerate(m.cfg.blocks):
            if b.experts and m.moe_key(i) not in self.moe:
                arena = m.layers[i]["arena"]
                mb = MoeBuffers()
                mb.alloc_moe(z, R, b.top, b.experts, b.experts + b.identity, arena.ef.H, arena.ef.F, tc=not m.f32, act_dtype=act)
                if mb.tc_ok:
                    mb.tc_xs = z(R * b.top, arena.ef.H, dtype=torch.float16)
                    mb.tc_act = z(R * b.top, arena.ef.F, dtype=torch.float16)
                self.moe[m.moe_key(i)] = mb
        self._delta = self._chunk = self._tmix = None

    def delta_scratch(self, b: BlockSpec, R: int, ra: int, rg: int, chunks: int):
        """Scratch of the row-parallel form of a delta-rule layer (grown on first use; decode steps never ask for it)."""
        n = int(nat.call("lsb_delta_scratch_floats", R, b.heads, b.dim, b.vdim, ra, rg))
        c = int(nat.call("lsb_delta_chunk_floats", chunks, b.heads, b.dim)) if chunks else 0
        if n < 0 or c < 0:
            raise RuntimeError("the step's delta-rule scratch exceeds 2^31 floats: use a smaller prefill chunk")
        if self._delta is None or self._delta.numel() < n:
            self._delta = torch.empty(n, dtype=torch.float32, device=self.dev)
        if c and (self._chunk is None or self._chunk.numel() < c):
            self._chunk = torch.empty(c, dtype=torch.float32, device=self.dev)
        return self._delta, self._chunk

    def tmix_scratch(self, b: BlockSpec, R: int, chunks: int, rank: int):
        """Scratch of the chunked form of a time-mixing layer (grown on first use)."""
        n = int(nat.call("lsb_tmix_scratch_floats", R, chunks, b.heads, b.dim, b.vdim, rank))
        if n < 0:
            raise RuntimeError("the step's time-mixing scratch exceeds 2^31 floats: use a smaller prefill chunk")
        if self._tmix is None or self._tmix.numel() < n:
            self._tmix = torch.empty(n, dtype=torch.float32, device=self.dev)
        return self._tmix


class BlockModel(ModelBase):
    mixed_steps = True

    def __init__(self, cfg: ModelConfig, device="cuda", kv_fmt: Optional[str] = None, page: int = 64, tp_rank: int = 0, tp_size: int = 1,
                 dtype: str = "bfloat16"):
        if tp_size != 1:
            raise NotImplementedError("models described layer by layer run on one GPU")
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {dtype!r}: bfloat16 or float32")
        self.f32 = dtype == "float32"
        fmt = "f32" if self.f32 else "bf16"
        if kv_fmt not in (None, fmt):
            logging.getLogger("layerstorm_b200.engine").info("kv format %s: this model keeps its attention cache in %s", kv_fmt, fmt)
        self._init_base(cfg, device, fmt, page, 0, 1)
        self.act_dtype = torch.float32 if self.f32 else torch.bfloat16
        self.w_fmt = "f32" if self.f32 else "bf16"
        self.expert_shard = "ep"
        self.Hp = _align(cfg.hidden, 8)
        self.zero, self._expand, self._expand_rows = torch.zeros(1, dtype=torch.int32, device=self.device), None, 0
        self.max_mix = 8
        mixing = [i for i, b in enumerate(cfg.blocks) if b.v_mix and b.kind == "attention"]
        self.v_first_layer = mixing[0] if mixing else -1
        if len({cfg.blocks[i].kv_heads * cfg.blocks[i].vdim for i in mixing}) > 1:
            raise ValueError("layers that mix values must have the same number of value channels")
        if cfg.residual_mult != 1.0 and not cfg.streams or cfg.streams and cfg.norm_place != "pre" or cfg.streams > 8 or cfg.streams and cfg.side_dim:
            raise ValueError("hyper-connections (up to 8 streams) come with norms in front of the sublayers, a residual factor comes with hyper-connections")
        if cfg.streams and (cfg.input_conv or cfg.loop) or cfg.loop and mixing or cfg.norm_place == "parallel" and any(b.branches for b in cfg.blocks) or cfg.input_conv > 17:
            raise ValueError("input convolutions (of up to 17 taps) and loops come with one residual stream, loops without value mixing, parallel sublayers with one mixer")
        if cfg.bigram and len(cfg.bigram) != 3:
            raise ValueError("a bigram embedding has a number of buckets and two multipliers")
        for i, b in [(i, m) for i, L in enumerate(cfg.blocks) for m in L.mixers]:
            if b.kind == "time_mix" and cfg.input_conv:
                raise ValueError(f"layer {i}: time mixing behind an input convolution")
            if b.heads % max(b.kv_heads, 1) or min(b.heads, b.kv_heads, b.dim, b.vdim) < 1:
                raise ValueError(f"layer {i}: {b.heads} heads over {b.kv_heads} groups of widths {b.dim} / {b.vdim}")
            if b.latent and (b.kv_rank < 1 or b.rot_dim < 0 or b.rot_dim % 2):
                raise ValueError(f"layer {i}: latent rows of {b.kv_rank} + {b.rot_dim} channels")
            if b.recurrent and b.dim > 256:
                raise ValueError(f"layer {i}: key heads of up to 256 channels, not {b.dim}")
        for i, b in enumerate(cfg.blocks):
            if b.experts and (b.top > min(32, b.experts + b.identity) or (b.experts + b.identity) % b.groups or b.groups > 64):
                raise ValueError(f"layer {i}: router with {b.experts} + {b.identity} outputs, top {b.top}, {b.groups} groups")

    @staticmethod
    def head_pad(d: int) -> int:
        return int(nat.call("lsb_attn_head_pad", d))

    @staticmethod
    def latent_pad(d: int) -> int:
        return _align(d, 16)

    def latent_row(self, b: BlockSpec) -> int:
        """Elements of a token's cached row (and of a head's query) in a latent layer."""
        return self.latent_pad(b.kv_rank) + self.latent_pad(b.rot_dim)

    def moe_key(self, i: int) -> tuple:
        b = self.cfg.blocks[i]
        return (b.experts, b.identity, b.top, b.ff)

    # ------------------------------------------------------------------ construction
    def _vec(self, t: torch.Tensor) -> torch.Tensor:
        return t.to(self.device).float().reshape(-1).contiguous()

    def _mat(self, *parts: torch.Tensor, cols: Optional[int] = None) -> QLinear:
        """Stacked projections as one matrix: every part padded to a multiple of 8 rows, the columns to ``cols`` (zeros)."""
        cols = cols or _align(parts[0].shape[1], 8)
        rows = [_align(p.shape[0], 8) for p in parts]
        w = torch.zeros(sum(rows), cols, dtype=self.act_dtype, device=self.device)
        r0 = 0
        for p, n in zip(parts, rows):
            w[r0: r0 + p.shape[0], : p.shape[1]] = p.to(self.device)
            r0 += n
        return QLinear(self.w_fmt, w.shape[0], cols, w)

    def _build_mixer(self, w, p: str, b: BlockSpec, M: dict):
        """Puts a mixer's device tensors into ``M``; returns the projections that read the layer's input as it is, and the output projection.
        ``M["meta"]`` counts columns from the first of these projections."""
        dev = self.device
        if b.delta:
            k = p + "kda."
            kw, vw = b.kv_heads * b.dim, b.heads * b.vdim
            low = b.kind == "channel_delta"
            parts = [w[k + n].to(dev) for n in (("q", "k", "v", "beta", "f_a", "g_a") if low else ("q", "k", "v", "beta", "a", "g"))]
            ra = rg = 0
            if low:
                fb, gb = w[k + "f_b"].to(dev), w[k + "g_b"].to(dev)
                ra, rg = _align(fb.shape[1], 8), _align(gb.shape[1], 8)
                pad = lambda t, n: torch.nn.functional.pad(t.float(), (0, n - t.shape[1])).to(self.act_dtype).contiguous()
                M["w_a"], M["w_g"] = pad(fb, ra), pad(gb, rg)
                if not self.f32:
                    # [W | W]: many rows take the low-rank products on the tensor cores with (hi | lo) activations
                    M["w_a2"], M["w_g2"] = torch.cat([M["w_a"]] * 2, 1).contiguous(), torch.cat([M["w_g"]] * 2, 1).contiguous()
            M["meta"] = _Meta(_offsets(parts), ra, rg)
            for n in ("conv_q", "conv_k", "conv_v"):
                t = w[k + n].to(dev).float().contiguous()
                if tuple(t.shape) != ((vw if n == "conv_v" else kw), b.conv):
                    raise ValueError(f"{k + n}: shape {tuple(t.shape)}")
                M[n] = t
            M["a_exp"], M["dt_bias"], M["o_norm"] = torch.exp(self._vec(w[k + "a_log"])), self._vec(w[k + "dt_bias"]), self._vec(w[k + "o_norm"]) * b.out_scale
            return parts, w[k + "o"].to(dev)
        if b.kind == "time_mix":
            k = p + "tmix."
            own = [w[k + n].to(dev) for n in ("r", "k", "v", "g", "w1")]
            M["shift"] = self._mat(*own, cols=self.Hp)
            M["meta"] = _Meta(_offsets(own))
            M["seg_rows"] = torch.tensor(M["meta"].offs, dtype=torch.int32)
            M["segs"] = [t.shape[0] for t in own]
            rank = _align(own[4].shape[0], 8)
            w2 = w[k + "w2"].to(dev)
            M["w2"] = torch.nn.functional.pad(w2.float(), (0, rank - w2.shape[1])).to(self.act_dtype).contiguous()
            M["w22"] = None if self.f32 else torch.cat([M["w2"]] * 2, 1).contiguous()
            mu = torch.zeros(5, self.Hp, device=dev)
            for j, n in enumerate("rkvgw"):
                mu[j, : self.cfg.hidden] = w[k + "mu_" + n].to(dev)
            M["mu"], M["w0"], M["u"], M["o_norm"] = mu, self._vec(w[k + "w0"]), self._vec(w[k + "u"]), self._vec(w[k + "o_norm"]) * b.out_scale
            return [], w[k + "o"].to(dev)
        a = p + "attn."
        if b.latent:
            own = b.kv_from < 0
            qn = "q_a" if b.q_rank else "q"
            names = [qn] + (["kv_a"] if own else []) + (["g"] if b.out_gate or b.head_gate else [])
            parts = [w[a + n].to(dev) for n in names]
            at = dict(zip(names, _offsets(parts)))
            M["meta"] = _Meta([at[qn], at.get("kv_a", -1), at.get("g", -1)])
            if b.q_rank:
                M["q_norm"], M["q_up"] = self._vec(w[a + "q_a_norm"]), self._mat(w[a + "q_b"].to(dev))
            dnp, dlp = _align(b.dim, 8), self.latent_pad(b.kv_rank)
            uk, uv = w[a + "k_b"].to(dev).view(b.heads, b.dim, b.kv_rank), w[a + "v_b"].to(dev).view(b.heads, b.vdim, b.kv_rank)
            M["w_uk"] = torch.zeros(b.heads, dlp, dnp, dtype=self.act_dtype, device=dev)
            M["w_uk"][:, : b.kv_rank, : b.dim] = uk.transpose(1, 2)
            M["w_uv"] = torch.zeros(b.heads, b.vdim, dlp, dtype=self.act_dtype, device=dev)
            M["w_uv"][:, :, : b.kv_rank] = uv
            if not self.f32:
                # the same two, one after the other per position: what long prompt runs make keys and values with
                dnw, dvp = _align(b.dim, 16), self.head_pad(b.vdim)
                M["w_kv"] = torch.zeros(b.heads * (dnw + dvp), dlp, dtype=self.act_dtype, device=dev)
                M["w_kv"][: b.heads * dnw].view(b.heads, dnw, dlp)[:, : b.dim, : b.kv_rank] = uk
                M["w_kv"][b.heads * dnw:].view(b.heads, dvp, dlp)[:, : b.vdim, : b.kv_rank] = uv
            if own:
                M["kv_norm"] = self._vec(w[a + "kv_a_norm"])
            M["inv_freq"] = self._inv_freq(b.rot_base, b.rot_dim)
            return parts, w[a + "o"].to(dev)
        gate = b.out_gate or b.head_gate
        names = ["q", "k"] + ([] if b.shared_kv else ["v"]) + (["g"] if gate else [])
        parts = [w[a + n].to(dev) for n in names]
        at = dict(zip(names, _offsets(parts)))
        M["meta"] = _Meta([at["q"], at["k"], at.get("v", at["k"]), at.get("g", -1)])       # shared keys and values: one projection
        for n in ("temp", "sink"):
            if getattr(b, n):
                M[n] = self._vec(w[a + n])
        if b.maps > 1:
            dot = lambda j: float((w[a + f"lq{j}"].double() * w[a + f"lk{j}"].double()).sum())
            M["lambda"] = math.exp(dot(1)) - math.exp(dot(2)) + b.diff
        if b.qkv_bias:
            M["q_bias"], M["k_bias"], M["v_bias"] = (self._vec(w[a + n + "_bias"]) for n in "qkv")
        if b.qk_norm or b.head_norm == "weight":
            M["q_norm"], M["k_norm"] = self._vec(w[a + "q_norm"]), self._vec(w[a + "k_norm"])
        if b.half_rot or b.pair_rot:
            M["inv_freq"] = self._inv_freq(b.rot_base, b.half_rot or b.pair_rot)
        if b.bias_rows:
            rel = w[a + "rel"].to(dev).float()                 # one value per distance and head: the kernels know no buckets
            M["bias"] = rel[torch.tensor(distance_buckets(rel.shape[0], b.bias_max), device=dev)].T.contiguous()
        if b.alibi:
            M["slope"] = torch.tensor([2.0 ** (-8.0 * (h + 1) / b.heads) for h in range(b.heads)], dtype=torch.float32, device=dev)
        if b.v_mix:
            M["v_mix"] = self._vec(w[a + "v_mix"])
        return parts, w[a + "o"].to(dev)

    def _inv_freq(self, base: float, dims: int) -> torch.Tensor:
        return torch.tensor([base ** (-2.0 * j / dims) for j in range(dims // 2)], dtype=torch.float64, device=self.device)

    @classmethod
    def from_state_dict(cls, cfg: ModelConfig, w, device="cuda", kv_fmt=None, page=64, expert_quant=None, dense_quant=None, tp_rank: int = 0,
                        tp_size: int = 1, expert_shard=None, with_mtp: bool = False, layer_hook=None, skip_experts=None, dtype: str = "bfloat16") -> "BlockModel":
        """Canonical state dict (any mapping with ``in`` and ``[]``) -> device model.  Quantised experts, tensor parallelism and expert
        streaming are not part of this model kind: ``expert_quant`` / ``dense_quant`` other than bf16, ``layer_hook`` are refused."""
        for q in (expert_quant, dense_quant):
            if q not in (None, "bf16", "f32"):
                raise NotImplementedError(f"weights of models described layer by layer are kept as they are, not in {q}")
        if layer_hook is not None:
            raise NotImplementedError("experts of models described layer by layer stay resident")
        m = cls(cfg, device, kv_fmt, page, tp_rank, tp_size, dtype)
        H, Hp, dev = cfg.hidden, m.Hp, m.device

        kind, sandwich = NORM_KIND[cfg.norm_kind], cfg.norm_place == "sandwich"

        def norm(p, scale=1.0):
            """(kind, weight, bias, alpha) of a norm of the residual stream"""
            b, al = p + ".bias", p + ".alpha"
            wt = m._vec(w[p + ".weight"]) * scale
            return kind, wt.expand(H).contiguous() if cfg.norm_scalar else wt, (m._vec(w[b]) * scale if b in w else None), (m._vec(w[al]) if al in w else None)

        def stacked(parts, cols=Hp):
            """The parts as one projection and the row at which each starts."""
            return m._mat(*parts, cols=cols), _offsets(parts)

        e = torch.zeros(cfg.vocab, Hp, dtype=torch.bfloat16, device=dev)
        e[:, :H] = w["embed.weight"].to(dev)
        m.embed = e
        hw = w["head.weight"].to(dev)
        m.head = m._mat(hw, cols=Hp)
        m.head.N = cfg.vocab                                   # padding rows of the matrix are never computed
        m.final_norm = norm("final_norm", cfg.logit_scale)     # the scale of the logits rides on the last norm
        if cfg.bigram:
            m.bigram = torch.zeros(cfg.bigram[0] + 1, Hp, dtype=torch.bfloat16, device=dev)
            m.bigram[:, :H] = w["bigram.weight"].to(dev)
        if cfg.loop:
            m.loop_step = torch.zeros(cfg.loop[2], Hp, device=dev)
            m.loop_step[:, :H] = w["loop_step"].to(dev)
        if cfg.side_dim:
            m.side_embed = w["side_embed.weight"].to(dev).to(torch.bfloat16).contiguous()
        for i, b in enumerate(cfg.blocks):
            p = f"layers.{i}."
            L: dict = {"mix_in": norm(p + "mix_norm"), "mix_out": norm(p + "mix_post_norm")} if sandwich else {"mix_in": NO_NORM, "mix_out": norm(p + "mix_norm")}
            if cfg.norm_place in ("pre", "parallel"):
                L["mix_in"], L["mix_out"] = L["mix_out"], NO_NORM
            if cfg.input_conv:
                taps = w[p + "input_conv"].to(dev)
                if tuple(taps.shape) != (H, cfg.input_conv):
                    raise ValueError(f"{p}input_conv: shape {tuple(taps.shape)}")
                L["conv_w"] = torch.zeros(cfg.input_conv, Hp, device=dev)
                L["conv_w"][:, :H] = taps.float().T
            sides, cols = _sides(b), 0
            L["sides"] = [{} for _ in sides]
            parts, outs, base = [], [], 0
            for (side, x), M in zip(sides, L["sides"]):
                own, out = m._build_mixer(w, p + side, x, M)
                if "shift" not in M:
                    M["meta"].shift(base)
                M["col"], M["cols"] = cols, _align(out.shape[1], 8)
                cols += M["cols"]
                base += sum(_align(t.shape[0], 8) for t in own)
                parts += own
                outs.append(out)
            # one norm for both sublayers: what the feed-forward projects with follows the mixer's projections, its way back is part of the mixer's
            both = cfg.norm_place == "parallel" and b.has_ff
            glu_ff = (b.dense_ff or b.shared_ff) if both else 0
            glu = ("mlp." if b.dense_ff else "moe.shared.0.") if glu_ff else ""
            ff_parts = []
            if both:
                ff_parts = ([w[p + "moe.router"].to(dev)] if b.experts else []) + ([w[p + glu + n].to(dev) for n in ("gate", "up")] if glu else [])
                ff_parts += [w[p + "moe.shared_gate"].to(dev)] if b.experts and b.shared_ff else []
            L["mix_ld"] = cols + _align(glu_ff, 8)
            L["glu_at"] = cols
            L["in"] = stacked(parts + ff_parts)[0] if parts + ff_parts else None
            if both:
                W, n = L["in"], sum(_align(t.shape[0], 8) for t in parts)
                L["halves"] = (QLinear(W.fmt, n, Hp, W.w[:n]), QLinear(W.fmt, W.N - n, Hp, W.w[n:]))
                L["half_rows"] = torch.tensor([0, n], dtype=torch.int32)
                L["ff_at"], L["ff_offs"] = n, [n + o for o in _offsets(ff_parts)]
                base += W.N - n
            for M in L["sides"]:
                if "shift" in M:                              # projections over inputs of their own, behind the others
                    M["meta"].shift(base)
                    M["at"] = base
                    base += M["shift"].N
            m.max_proj = max(m.max_proj, base)
            if b.branches and b.join == "normed":
                for (side, _), M, t in zip(sides, L["sides"], outs):
                    M["out"], M["out_norm"] = m._mat(t, cols=M["cols"]), m._vec(w[p + side + "out_norm"])
                    M["out"].N = Hp
            else:
                pad = torch.nn.functional.pad
                wide = [pad(t, (0, M["cols"] - t.shape[1])) for t, M in zip(outs, L["sides"])]
                if glu:
                    t = w[p + glu + "down"].to(dev)
                    wide.append(pad(t, (0, _align(t.shape[1], 8) - t.shape[1])))
                L["out"] = m._mat(torch.cat(wide, 1))
                L["out"].N = Hp
            m.max_mix = max(m.max_mix, L["mix_ld"])
            if cfg.streams:
                for q in ["mix_hc"] + (["ffn_hc"] if b.has_ff else []):
                    L[q] = tuple(m._vec(w[f"{p}{q}.{k}"]) for k in ("in", "out", "mix"))
            if b.has_ff and not both:
                L["ff_in"], L["ff_out"] = (norm(p + "ffn_norm"), norm(p + "ffn_post_norm")) if sandwich else (NO_NORM, norm(p + "ffn_norm"))
                if cfg.norm_place == "pre":
                    L["ff_in"], L["ff_out"] = L["ff_out"], NO_NORM
            if b.dense_ff and not both:
                L["ff"], L["ff_offs"] = stacked([w[p + f"mlp.{n}"].to(dev) for n in ("gate", "up")])
                L["ff_down"] = m._mat(w[p + "mlp.down"].to(dev))
                L["ff_down"].N = Hp
                m.max_proj = max(m.max_proj, L["ff"].N)
            if b.experts:
                mo = p + "moe."
                # the router and - where there is one - the shared expert's gate, up and output-gate rows are one product (values of the file's
                # type: fp32-accumulated products are exact in them)
                if not both:
                    parts = [w[mo + "router"].to(dev)] + ([w[mo + n].to(dev) for n in ("shared.0.gate", "shared.0.up", "shared_gate")] if b.shared_ff else [])
                    L["router"], L["ff_offs"] = stacked(parts)
                    m.max_proj = max(m.max_proj, L["router"].N)
                    if b.shared_ff:
                        L["ff_down"] = m._mat(w[mo + "shared.0.down"].to(dev))
                        L["ff_down"].N = Hp
                L["router_bias"] = m._vec(w[mo + "router_bias"]) if (b.correction or b.logit_bias) and (mo + "router_bias") in w else None
                # expert width padded to the tensor-core tile where the residual width allows that path
                F = _align(b.ff, 128) if Hp % 128 == 0 else _align(b.ff, 8)
                gated = b.unit == "glu"
                arena = ExpertArena(expert_layout(m.w_fmt, Hp, F, gated=gated), b.experts, b.experts, dev)
                for x in range(b.experts):
                    u, d = (torch.zeros(n, k, dtype=m.act_dtype, device=dev) for n, k in ((F, Hp), (Hp, F)))
                    u[: b.ff, :H], d[:H, : b.ff] = (w[mo + f"experts.{x}.{n}"].to(dev) for n in ("up", "down"))
                    g = None
                    if gated:
                        g = torch.zeros_like(u)
                        g[: b.ff, :H] = w[mo + f"experts.{x}.gate"].to(dev)
                        g = QLinear(m.w_fmt, F, Hp, g)
                    arena.write_expert(x, g, QLinear(m.w_fmt, F, Hp, u), QLinear(m.w_fmt, Hp, F, d))
                    arena.slot_of[x] = x
                L["arena"] = arena
            if cfg.side_dim:
                L["side_gate"] = m._mat(w[p + "side.gate"].to(dev), cols=Hp)
                L["side_proj"] = m._mat(w[p + "side.proj"].to(dev))
                L["side_proj"].N = Hp
                L["side_norm"] = (NORM_KIND["rms"], m._vec(w[p + "side.norm"]), None, None)
                m.max_proj = max(m.max_proj, L["side_gate"].N)
            m.layers.append(L)
        m.max_proj, m.max_mix = _align(m.max_proj, 8), _align(m.max_mix, 8)
        return m

    @classmethod
    def random_init(cls, cfg: ModelConfig, device="cuda", kv_fmt=None, page=64, seed=0, expert_slots=None, embed_on_host: bool = False,
                    reserve_bytes: int = 0, tp_rank: int = 0, tp_size: int = 1, expert_shard=None, with_mtp: bool = False, layer_hook=None,
                    dtype: str = "bfloat16") -> "BlockModel":
        """Random weights made on the device, tensor by tensor."""
        return cls.from_state_dict(cfg, RandomBlockWeights(cfg, seed, device), device, kv_fmt, page, tp_rank=tp_rank, tp_size=tp_size,
                                   layer_hook=layer_hook, dtype=dtype)

    # ------------------------------------------------------------------ caches and workspaces
    def make_workspace(self, R: int, n_logit_rows: int, max_ctx: int) -> BlockWorkspace:
        return BlockWorkspace(self, R, n_logit_rows, max_ctx)

    def alloc_cache(self, num_pages: int, n_slots: int, max_pages_per_seq: int):
        self.num_pages, self.n_slots, self.max_pages = num_pages, n_slots, max_pages_per_seq
        z = lambda *s, dtype=torch.float32: torch.zeros(*s, dtype=dtype, device=self.device)
        self.block_table = z(n_slots, max_pages_per_seq, dtype=torch.int32)
        self.idx_block_table = self.block_table
        runs = self.cfg.layer_runs()
        if self.cfg.input_conv > 1:
            for k in range(len(runs)):                                      # the inputs that the run's convolution looks back at
                self.kda_conv["input", k] = z(n_slots, self.cfg.input_conv - 1, self.Hp)
        for i, b in [(k, m) for k, (i, _) in enumerate(runs) for m in self.cfg.blocks[i].mixers]:
            if b.delta:
                self.kda_state[i] = z(n_slots, b.heads, b.vdim, int(nat.call("lsb_delta_key_pad", b.dim)))
                self.kda_conv[i] = z(n_slots, b.heads, 2 * b.dim + b.vdim, b.conv - 1)
            elif b.kind == "time_mix":
                self.kda_state[i] = z(n_slots, b.heads, b.vdim, int(nat.call("lsb_tmix_key_pad", b.dim)))
                self.kda_conv[i] = z(n_slots, self.Hp)                   # the previous token's input
            elif b.latent:
                if b.kv_from < 0:
                    self.kv_cache[i] = z(num_pages, self.page, self.latent_row(b), dtype=self.act_dtype)
            else:
                self.kv_cache[i] = z(num_pages, self.page, b.kv_heads * (b.maps * self.head_pad(b.dim) + self.head_pad(b.vdim)), dtype=self.act_dtype)

    def cache_bytes_per_token(self) -> int:
        width = lambda b: ((self.latent_row(b) if b.kv_from < 0 else 0) if b.latent else b.kv_heads * (b.maps * self.head_pad(b.dim) + self.head_pad(b.vdim)))
        return sum(width(b) * (4 if self.f32 else 2) for i, _ in self.cfg.layer_runs() for b in self.cfg.blocks[i].mixers if not b.recurrent)

    # ------------------------------------------------------------------ forward
    def _resid_rows(self, ws, R: int, H: int) -> torch.Tensor:
        return ws.streams[:R, :, :H].sum(1) if self.cfg.streams else ws.resid[:R, :H]

    def _mixer(self, k: int, i: int, b: BlockSpec, L: dict, ws: BlockWorkspace, R: int, nseq: int):
        """The mixers of layer i in its run k, input projections to output projection: ``ws.sub`` (and ``ws.sub2`` of a second result that is normed on its
        own).  With both sublayers on one norm the feed-forward's projections and gated unit as well: all of the layer but its routed experts."""
        if "halves" in L:
            self._project_both(L, ws, R)
        elif L["in"] is not None:
            L["in"](ws.proj, ws.x_mix, R, ldo=self.max_proj)
        for x, M in zip(b.mixers, L["sides"]):
            f = self._delta if x.delta else (self._time_mix if x.kind == "time_mix" else (self._latent if x.latent else self._attention))
            f(k, i, x, M, ws, R, nseq, ws.mix.view(-1)[M["col"]:], L["mix_ld"])
        if "halves" in L and (b.dense_ff or b.shared_ff):
            ff = b.dense_ff or b.shared_ff
            g, u, s = (*L["ff_offs"], -1) if b.dense_ff else L["ff_offs"][1:]
            nat.call("lsb_glu", ws.mix.view(-1)[L["glu_at"]:], L["mix_ld"], _align(ff, 8), ws.proj, self.max_proj, g, u, s, R, ff, 0.0 if b.dense_ff else b.shared_limit,
                     *((1.0, 0.0) if b.dense_ff else (b.act_alpha, b.act_shift)), int(self.f32))
        if b.branches and b.join == "normed":
            for M, sub in zip(L["sides"], (ws.sub, ws.sub2)):
                M["out"](sub, ws.mix.view(-1)[M["col"]:], R, ldx=L["mix_ld"], ldo=self.Hp)
        else:
            L["out"](ws.sub, ws.mix, R, ldo=self.Hp)

    def _project_both(self, L: dict, ws: BlockWorkspace, R: int):
        """The mixer's projections (of its own input) and the feed-forward's (of the norm as it is), side by side in ``ws.proj``."""
        W, (mix, ff) = L["in"], L["halves"]
        if ws.x_pair is None:
            W(ws.proj, ws.x, R, ldo=self.max_proj)
        elif not self.f32 and R < 8 and self.Hp <= 16384:
            nat.call("lsb_gemv_bf16_segs", ws.proj, ws.x_pair, W.w, R, W.N, self.Hp, self.Hp, self.Hp, self.max_proj, L["half_rows"], 2, ws.x_pair.stride(0))
        else:
            mix(ws.proj, ws.x_mix, R, ldo=self.max_proj)
            ff(ws.proj.view(-1)[L["ff_at"]:], ws.x, R, ldo=self.max_proj)

    def _attention(self, k: int, i: int, b: BlockSpec, M: dict, ws: BlockWorkspace, R: int, nseq: int, out, ldo: int):
        dkp, dvp, ldp = self.head_pad(b.dim), self.head_pad(b.vdim), self.max_proj
        oq, ok, ov, og = M["meta"].offs
        H, G = b.heads * b.maps, b.kv_heads * b.maps
        at = (ws.q, self.kv_cache[k], self.block_table, self.max_pages, ws.row_seq, ws.row_pos, R, H, G, b.dim, b.vdim, dkp, dvp, self.page, int(self.f32))
        if b.qkv_bias or b.head_norm or b.half_rot or b.pair_rot or b.temp or b.shared_kv or b.maps > 1:
            nat.call("lsb_attn_head_prep", ws.proj, ldp, oq, ok, ov, M.get("q_bias"), M.get("k_bias"), M.get("v_bias"), HEAD_NORM[b.head_norm], M.get("q_norm"),
                     M.get("k_norm"), self.cfg.rms_eps, b.half_rot or b.pair_rot, int(b.pair_rot > 0), M.get("inv_freq"), M.get("temp"), b.maps, *at)
        else:
            mix = 0 if not b.v_mix else (1 if i == self.v_first_layer else 2)
            nat.call("lsb_attn_prep", ws.proj, ldp, oq, ok, ov, M.get("q_norm"), M.get("k_norm"), self.cfg.rms_eps, ws.v_first if mix else None, mix, M.get("v_mix"), *at)
        bias, run = M.get("bias"), max(ws.seq_rows)
        nat.call("lsb_attn", ws.q, self.kv_cache[k], self.block_table, self.max_pages, self.page, ws.row_seq, ws.row_pos, ws.seq_row0, ws.seq_nrows, nseq,
                 run, ws.proj, ldp, og, out, ldo, ws.o_part, ws.ml_part, ws.splits[i], R, H, G, b.dim, b.vdim, dkp, dvp,
                 b.window, b.scale, M.get("slope"), int(b.head_gate), b.chunk, bias, bias.shape[1] if bias is not None else 0, b.out_scale, M.get("sink"), b.maps,
                 int(self.f32))
        if b.maps > 1:
            n = nat.call("lsb_attn_partials", run, H, G, dkp, dvp, ws.splits[i], int(self.f32))
            nat.call("lsb_attn_diff", out, ldo, ws.o_part, ws.ml_part, n, R, b.heads, b.heads // b.kv_heads, b.vdim, dvp, M["lambda"], self.cfg.rms_eps,
                     b.out_scale * (1.0 - b.diff), ws.row_seq, int(self.f32))

    def _latent(self, k: int, i: int, b: BlockSpec, L: dict, ws: BlockWorkspace, R: int, nseq: int, out, ldo: int):
        cache = self.kv_cache[k if b.kv_from < 0 else b.kv_from]
        q, ldq = ws.proj.view(-1)[L["meta"].offs[0]:], self.max_proj           # the heads' queries: straight from the projection or through a latent
        if b.q_rank:
            nat.call("lsb_norm_rows", ws.q_low, L["q_up"].K, q, ldq, None, 0, L["q_norm"], None, None, R, b.q_rank, self.cfg.rms_eps, NORM_KIND["rms"], int(self.f32))
            q, ldq = ws.q_up, L["q_up"].N
            L["q_up"](q, ws.q_low, R)
        # long runs one by one, what lies between them together
        rows, row0, j = ws.seq_rows, 0, 0
        while j < nseq:
            e, n = j + 1, rows[j]
            at = (q[row0 * ldq:], ldq)
            if self._expands(b, rows[j], ws.seq_end[j]):
                self._latent_run(b, L, ws, cache, *at, row0, n, j, out, ldo)
            else:
                while e < nseq and not self._expands(b, rows[e], ws.seq_end[e]):
                    n, e = n + rows[e], e + 1
                self._latent_rows(i, b, L, ws, cache, *at, row0, n, j, e, out, ldo)
            row0, j = row0 + n, e

    def _latent_rows(self, i: int, b: BlockSpec, L: dict, ws: BlockWorkspace, cache, qsrc, ldq: int, r0: int, R: int, j: int, k: int, out, ldo: int):
        """Step rows [r0, r0 + R) (sequences j .. k - 1 of the step) in the latent space."""
        _, okv, og = L["meta"].offs
        H, ld, f32, err = b.heads, self.max_proj, int(self.f32), TcScratch.get(self.device).err
        ag = -1 if b.out_gate else og                          # a gate per head acts on the latent sums, one per value channel on the result
        q, o_lat, proj, seq, pos = ws.q_lat[r0 * H * self.latent_row(b):], ws.o_lat[r0 * H * L["w_uv"].shape[2]:], ws.proj[r0:], ws.row_seq[r0:], ws.row_pos[r0:]
        nat.call("lsb_latent_query", qsrc, ldq, proj, ld, okv, L.get("kv_norm"), self.cfg.rms_eps, L["inv_freq"], L["w_uk"], q, ws.q_nope, cache, self.block_table,
                 self.max_pages, self.page, seq, pos, R, H, b.dim, L["w_uk"].shape[2], b.rot_dim, b.kv_rank, f32, err)
        # seq_row0 holds row numbers of the step, so runs get the whole buffers (steps with key splits have no long runs: r0 is 0)
        run = max(ws.seq_rows[j:k])
        rows = (q, proj, seq, pos, o_lat) if run == 1 else (ws.q_lat, ws.proj, ws.row_seq, ws.row_pos, ws.o_lat)
        nat.call("lsb_latent_attn", rows[0], cache, self.block_table, self.max_pages, self.page, rows[2], rows[3], ws.seq_row0[j:], ws.seq_nrows[j:], k - j, run,
                 rows[1], ld, ag, rows[4], ws.lat_o_part, ws.lat_ml_part, ws.lat_splits[i], R, H, b.kv_rank, b.rot_dim, b.window, b.scale, f32)
        nat.call("lsb_latent_out", out[r0 * ldo:], ldo, o_lat, ws.lat_o_part, ws.lat_ml_part, ws.lat_parts[i], L["w_uv"], proj, ld, og, int(b.head_gate), seq, R, H,
                 b.kv_rank, b.vdim, f32, err)

    def _latent_run(self, b: BlockSpec, L: dict, ws: BlockWorkspace, cache, qsrc, ldq: int, r0: int, R: int, j: int, out, ldo: int):
        """Step rows [r0, r0 + R), a run of sequence j, over keys and values of every head, made for this step from the cached rows that the run sees."""
        _, okv, og = L["meta"].offs
        H, ld, err, T = b.heads, self.max_proj, TcScratch.get(self.device).err, ws.seq_end[j]
        dnw, dvp, drp = _align(b.dim, 16), self.head_pad(b.vdim), self.latent_pad(b.rot_dim)
        base = self._first_seen(b, R, T)
        Tm, proj, seq, pos = _align(T - base, 256), ws.proj[r0:], ws.row_seq[r0:], ws.row_pos[r0:]
        q, lat, kv = self._expand_scratch(ws.R, R * H * (dnw + drp), Tm * self.latent_pad(b.kv_rank), Tm * (H * (dnw + dvp) + drp))
        nat.call("lsb_latent_expand", qsrc, ldq, proj, ld, okv, L.get("kv_norm"), self.cfg.rms_eps, L["inv_freq"], L["w_kv"], q, lat, kv, cache, self.block_table,
                 self.max_pages, self.page, seq, pos, R, base, T, Tm, H, b.dim, dnw, b.rot_dim, b.kv_rank, dvp, err)
        nat.call("lsb_attn_run", q, kv, Tm, self.zero, seq, pos, self.zero, ws.seq_nrows[j:], proj, ld, og, int(b.head_gate), out[r0 * ldo:], ldo, R, H, dnw, drp, b.vdim,
                 dvp, b.window, base, b.scale)

    @staticmethod
    def _first_seen(b: BlockSpec, R: int, T: int) -> int:
        """First position that any of the last R of T positions sees."""
        return max(0, T - R - b.window + 1) if b.window else 0

    def _expands(self, b: BlockSpec, R: int, T: int) -> bool:
        """Whether a run of R rows over T positions is worth writing keys and values out for (and the kernels take the sizes): fewer operations per
        (query, key), against a product over all positions that runs about four times as fast per operation."""
        dnw, dvp = _align(b.dim, 16), self.head_pad(b.vdim)
        row, T = b.heads * (dnw + dvp) + self.latent_pad(b.rot_dim), T - self._first_seen(b, R, T)
        return (not self.f32 and R >= EXPAND_ROWS and dnw + self.latent_pad(b.rot_dim) <= 256 and dvp <= 256 and 2 * T * row <= EXPAND_BYTES
                and R * (2 * b.kv_rank - b.dim - b.vdim) * 4 > (b.dim + b.vdim) * b.kv_rank)

    def _expand_scratch(self, R: int, *sizes: int) -> list:
        """bf16 scratch of long prompt runs, shared by the layers: made once, for the most rows and positions such runs can have."""
        if self._expand is None or R > self._expand_rows:
            need = 0
            for b in self.cfg.blocks:
                if b.latent:
                    dnw, drp, dlp = _align(b.dim, 16), self.latent_pad(b.rot_dim), self.latent_pad(b.kv_rank)
                    row = b.heads * (dnw + self.head_pad(b.vdim)) + drp
                    T = _align(min(self.max_pages * self.page, EXPAND_BYTES // (2 * row)), 256)
                    need = max(need, R * b.heads * (dnw + drp) + T * (dlp + row))
            self._expand, self._expand_rows = torch.empty(need + 192, dtype=torch.bfloat16, device=self.device), R
        at = [0]
        for n in sizes:
            at.append(at[-1] + _align(n, 64))
        return [self._expand[a: a + n] for a, n in zip(at, sizes)]

    def _delta(self, k: int, i: int, b: BlockSpec, L: dict, ws: BlockWorkspace, R: int, nseq: int, out, ldo: int):
        mt = L["meta"]
        rows = ws.seq_rows
        few = max(rows) <= FEW_ROWS and b.vdim <= nat.call("lsb_delta_few_max_dv", b.dim)
        scratch = chunk_ws = None
        long_, chunks = [], 0
        if not few:
            long_ = [n for n in rows if n >= LONG_ROWS] if b.dim <= 128 else []
            chunks = sum((n + 63) // 64 for n in long_)
            scratch, chunk_ws = ws.delta_scratch(b, R, mt.ra, mt.rg, chunks)
        oq, ok, ov, ob, oa, og = mt.offs
        nat.call("lsb_delta_forward", ws.proj, self.max_proj, oq, ok, ov, ob, oa, og, mt.ra, mt.rg, L.get("w_a"), L.get("w_g"), L.get("w_a2"), L.get("w_g2"),
                 L["conv_q"], L["conv_k"], L["conv_v"], L["a_exp"], L["dt_bias"], L["o_norm"], self.kda_state[k], self.kda_conv[k], ws.seq_row0,
                 ws.seq_nrows, ws.seq_slot, out, ldo, nseq, R, b.heads, b.kv_heads, b.dim, b.vdim, b.conv, 0 if b.decay == "softplus" else 1,
                 b.dim ** -0.5, b.decay_bound, self.cfg.rms_eps, int(self.f32), int(few), scratch, len(rows) - len(long_), len(long_), chunks, LONG_ROWS,
                 chunk_ws, TcScratch.get(self.device).err)

    def _time_mix(self, k: int, i: int, b: BlockSpec, M: dict, ws: BlockWorkspace, R: int, nseq: int, out, ldo: int):
        W, Hp, ldp, f32, err = M["shift"], self.Hp, self.max_proj, int(self.f32), TcScratch.get(self.device).err
        seqs = (ws.seq_row0, ws.seq_nrows, ws.seq_slot)
        nat.call("lsb_tmix_shift", ws.x, Hp, self.kda_conv[k], M["mu"], ws.xs, ws.xs.stride(0), *seqs, nseq, R, f32)
        r, segs = M["seg_rows"].tolist(), M["segs"]
        proj = ws.proj.view(-1)[M["at"]:]
        if not f32 and R < 8 and Hp <= 16384:
            nat.call("lsb_gemv_bf16_segs", proj, ws.xs, W.w, R, W.N, Hp, Hp, Hp, ldp, M["seg_rows"], 5, ws.xs.stride(0))
        elif not f32 and R >= 8 and len(set(segs[:4])) == 1:
            nat.call("lsb_gemm_bf16_tc_batched", proj, ws.xs, W.w, R, r[1], Hp, 4, Hp, ws.xs.stride(0), Hp, r[1] * Hp, ldp, r[1], 0, err)
            QLinear(W.fmt, W.N - r[4], Hp, W.w[r[4]:])(proj[r[4]:], ws.xs[4], R, ldo=ldp)
        else:
            for j, end in enumerate(r[1:] + [W.N]):
                QLinear(W.fmt, end - r[j], Hp, W.w[r[j]:])(proj[r[j]:], ws.xs[j], R, ldo=ldp)
        few = max(ws.seq_rows) <= FEW_ROWS or b.dim > 128
        rank = M["w2"].shape[1]
        chunks = 0 if few else sum((n + 63) // 64 for n in ws.seq_rows)
        scratch = None if few else ws.tmix_scratch(b, R, chunks, rank)
        nat.call("lsb_tmix_forward", ws.proj, ldp, *M["meta"].offs, rank, M["w2"], M["w22"], M["w0"], M["u"], M["o_norm"], self.kda_state[k], self.kda_conv[k], ws.x, Hp,
                 *seqs, out, ldo, nseq, R, b.heads, b.dim, b.vdim, self.cfg.rms_eps, f32, int(few), scratch, chunks, err)

    def _glu(self, L: dict, ws: BlockWorkspace, R: int, ff: int, offs, limit=0.0, alpha=1.0, shift=0.0):
        """Gated unit over columns of the projection in ``ws.proj`` and its down product into ``ws.sub``; ``offs``: gate, up, output gate (-1: none)."""
        K = L["ff_down"].K
        nat.call("lsb_glu", ws.glu, K, K, ws.proj, self.max_proj, *offs, R, ff, limit, alpha, shift, int(self.f32))
        L["ff_down"](ws.sub, ws.glu, R, ldo=self.Hp)

    def _moe(self, i: int, b: BlockSpec, L: dict, ws: BlockWorkspace, R: int) -> MoeBuffers:
        mb, cfg = ws.moe[self.moe_key(i)], self.cfg
        n = b.experts + b.identity
        both = "halves" in L                                   # then the router's logits and the shared expert stand where _mixer put them
        if not both:
            L["router"](ws.proj, ws.x, R, ldo=self.max_proj)
        nat.call("lsb_router_topk_grouped", ws.proj.view(-1)[L["ff_offs"][0]:], L["router_bias"], mb.ids, mb.wts, R, n, b.top, b.groups, b.keep,
                 LOGIT_SCORES if b.logit_bias else SCORING[b.scoring], int(cfg.norm_topk_prob), cfg.routed_scale, 0, self.max_proj, 1)
        if b.shared_ff and not both:
            self._glu(L, ws, R, b.shared_ff, L["ff_offs"][1:], b.shared_limit, b.act_alpha, b.act_shift)
        self.moe_prepare(L["arena"], mb, ws.x, R, b.experts)
        plain = b.act_alpha == 1.0 and b.act_shift == 0.0 and not b.scale_input
        act = "relu2" if b.unit == "relu2" else None if plain else (b.act_alpha, b.act_shift, mb.wts if b.scale_input else None)
        self.moe_experts(L["arena"], mb, ws.x, R, b.experts, b.limit, mb.miss, act)
        return mb

    def _update(self, ws: BlockWorkspace, R: int, post: tuple, pre: tuple, sub=None, mb: Optional[MoeBuffers] = None, b: Optional[BlockSpec] = None,
                L: Optional[dict] = None, run: Optional[tuple] = None):
        """resid += post(sub + expert sum), x = pre(resid).  ``run`` = (number, layer, pass that starts in front of it or -1): the layer run that follows
        reads x - through its convolution, and behind the vector of its pass."""
        Hp, y = self.Hp, (None, None, None, None, 0, 0, 0)
        if mb is not None:
            y = (mb.y, None if b.scale_input else mb.wts, mb.ids, L["arena"].slot_of, b.top, b.experts, L["arena"].ef.H)
        step, conv, taps = None, (None, None, None, None), 0
        if run is not None:
            k, i, t = run
            step, taps = self.loop_step[t] if t >= 0 else None, self.cfg.input_conv
        single = taps and pre[0] in (NORM_KIND["rms"], NORM_KIND["layer"]) and max(ws.seq_rows) == 1
        if taps:
            w, state = self.layers[i]["conv_w"], self.kda_conv.get(("input", k))
            if single:
                conv = (ws.x_mix, w, state, ws.row_seq)
        nat.call("lsb_resid_update", ws.x, Hp, ws.resid, Hp, sub, Hp, *post, *pre, R, self.cfg.hidden, self.cfg.rms_eps, *y, step, *conv, taps, Hp, int(self.f32))
        if taps and not single:
            nat.call("lsb_input_conv", ws.x_mix, ws.x, Hp, w, state, taps, Hp, ws.seq_row0, ws.seq_nrows, ws.seq_slot, len(ws.seq_rows), R, Hp, int(self.f32))

    def _side(self, i: int, L: dict, ws: BlockWorkspace, R: int):
        """The layer's per-token input: gate product on the stream, table slice, projection into ``ws.sub``."""
        d, K = self.cfg.side_dim, L["side_proj"].K
        L["side_gate"](ws.proj, ws.x, R, ldo=self.max_proj)
        nat.call("lsb_side_gate", ws.side, K, ws.proj, self.max_proj, self.side_embed, self.side_embed.shape[1], i * d, d, ws.tok, self.cfg.vocab, R, int(self.f32))
        L["side_proj"](ws.sub, ws.side, R, ldo=self.Hp)

    def set_layer_skip(self, skip=(), probe: bool = False):
        if probe:
            raise NotImplementedError("layer-input similarity probing is built for the MLA family")
        keep = {self.v_first_layer} | {b.kv_from for b in self.cfg.blocks}          # layers whose values or cached rows others read
        keep |= set(range(*self.cfg.loop[:2])) if self.cfg.loop else set()          # layers that run several times
        super().set_layer_skip([l for l in skip if int(l) not in keep], False)

    def forward(self, ws: BlockWorkspace, R: int, nseq: int, logit_row0: int, n_logit_rows: int):
        """One step over the first ``R`` staged rows; logits of rows [logit_row0, logit_row0 + n_logit_rows)."""
        cfg, H, Hp, f32 = self.cfg, self.cfg.hidden, self.Hp, int(self.f32)
        run = [i for i in range(cfg.n_layers) if i not in self.skip_layers]
        if cfg.streams:
            self._forward_streams(ws, R, nseq, run)
            if n_logit_rows:
                self.emit_logits(ws, logit_row0, n_logit_rows)
            return
        runs = [(k, i, t) for k, (i, t) in enumerate(cfg.layer_runs())]
        live = [r for r in runs if r[1] not in self.skip_layers]
        follows = dict(zip([-1] + [k for k, _, _ in live], live + [None]))       # the layer run that follows, and the norm in front of it
        enters = {k: self.layers[r[1]]["mix_in"] if r else NO_NORM for k, r in follows.items()}
        plain = enters[-1] is NO_NORM and not cfg.bigram and not cfg.input_conv and follows[-1][2] < 0
        if cfg.bigram:
            nat.call("lsb_embedding_bigram", ws.resid, self.embed, self.bigram, ws.tok, ws.prev_tok, R, Hp, cfg.vocab, cfg.embed_scale, *cfg.bigram)
        else:
            nat.call("lsb_embedding_scaled", ws.resid, ws.x if plain and not f32 else None, self.embed, ws.tok, R, Hp, 0, cfg.vocab, cfg.embed_scale)
        if not plain or f32:
            self._update(ws, R, NO_NORM, enters[-1], run=follows[-1])
        for k, i, _ in runs:
            if self.aux_capture is not None and all(j != i for _, j, _ in runs[:k]):
                self._capture_aux(i, ws, R)
            if k not in enters:
                continue
            b, L = cfg.blocks[i], self.layers[i]
            self._mixer(k, i, b, L, ws, R, nseq)
            last, nxt = (NO_NORM, None) if cfg.side_dim else (enters[k], follows[k])
            if cfg.norm_place == "parallel":
                self._update(ws, R, NO_NORM, last, ws.sub, self._moe(i, b, L, ws, R) if b.experts else None, b, L, run=nxt)
            else:
                self._update(ws, R, L["mix_out"], L["ff_in"] if b.has_ff else last, ws.sub, run=None if b.has_ff else nxt)
                if b.experts:
                    mb = self._moe(i, b, L, ws, R)
                    self._update(ws, R, L["ff_out"], last, ws.sub if b.shared_ff else None, mb, b, L, run=nxt)
                elif b.dense_ff:
                    L["ff"](ws.proj, ws.x, R, ldo=self.max_proj)
                    self._glu(L, ws, R, b.dense_ff, (*L["ff_offs"], -1))
                    self._update(ws, R, L["ff_out"], last, ws.sub, run=nxt)
            if cfg.side_dim:
                self._side(i, L, ws, R)
                self._update(ws, R, L["side_norm"], enters[k], ws.sub, run=follows[k])
            if self.drift is not None:
                step = self.loop_step[follows[k][2], :H] if follows[k] and follows[k][2] >= 0 else 0.0       # already on the stream, not yet the layer's
                self.drift[f"layer{k:03d}.resid"] = (ws.resid[:R, :H] - step).float().cpu()
        if self.aux_capture is not None:
            self._capture_aux(cfg.n_layers, ws, R)
        if n_logit_rows:
            self.emit_logits(ws, logit_row0, n_logit_rows)

    def _forward_streams(self, ws: BlockWorkspace, R: int, nseq: int, run: List[int]):
        """The layers of a model with hyper-connections; leaves the sum of the streams in ``ws.resid``."""
        cfg = self.cfg
        subs = [(i, q) for i in run for q in ("mix", "ffn") if q == "mix" or cfg.blocks[i].has_ff]
        enters = [(self.layers[i][q + "_hc"][0], self.layers[i]["mix_in" if q == "mix" else "ff_in"]) for i, q in subs] + [(None, NO_NORM)]
        nat.call("lsb_embedding_scaled", ws.resid, None, self.embed, ws.tok, R, self.Hp, 0, cfg.vocab, cfg.embed_scale)
        self._update_streams(ws, R, enters[0], first=ws.resid)
        for (i, q), nxt in zip(subs, enters[1:]):
            b, L = cfg.blocks[i], self.layers[i]
            if q == "mix" and self.aux_capture is not None:
                self._capture_aux(i, ws, R)
            mb = None
            if q == "mix":
                self._mixer(i, i, b, L, ws, R, nseq)
            elif b.experts:
                mb = self._moe(i, b, L, ws, R)
            else:
                L["ff"](ws.proj, ws.x, R, ldo=self.max_proj)
                self._glu(L, ws, R, b.dense_ff, (*L["ff_offs"], -1))
            self._update_streams(ws, R, nxt, L[q + "_hc"], None if mb is not None and not b.shared_ff else ws.sub, mb, b, L, q == "mix" and b.join == "normed" and b.branches)
            if self.drift is not None and (q == "ffn" or not b.has_ff):
                self.drift[f"layer{i:03d}.resid"] = self._resid_rows(ws, R, cfg.hidden).float().cpu()
        if self.aux_capture is not None:
            self._capture_aux(cfg.n_layers, ws, R)

    def _update_streams(self, ws: BlockWorkspace, R: int, nxt: tuple, hc: tuple = (None, None, None), sub=None, mb: Optional[MoeBuffers] = None, b=None, L=None,
                        normed=False, first=None):
        """Streams behind a sublayer with the weights ``hc``, and the input of the next one ``nxt`` = (its reading weights, its norm); behind the last
        (reading weights None) the sum of the streams instead."""
        Hp, y, last = self.Hp, (None, None, None, None, 0, 0, 0), nxt[0] is None
        if mb is not None:
            y = (mb.y, None if b.scale_input else mb.wts, mb.ids, L["arena"].slot_of, b.top, b.experts, L["arena"].ef.H)
        sides = ([ws.sub2, Hp] + [M["out_norm"] for M in L["sides"]]) if normed else [None, Hp, None, None]
        nat.call("lsb_stream_update", None if last else ws.x, Hp, ws.streams, Hp, self.cfg.streams, first, ws.resid if last else None, sub, *sides, hc[2], hc[1],
                 self.cfg.residual_mult, nxt[0], *nxt[1], R, self.cfg.hidden, self.cfg.rms_eps, *y, int(self.f32))

    def emit_logits(self, ws: BlockWorkspace, row0: int, n: int, rows: Optional[torch.Tensor] = None):
        """Logits of step rows [row0, row0 + n), or of the ``n`` rows listed in ``rows`` (int32, device), after :meth:`forward`."""
        kind, nw, nb, alpha = self.final_norm
        nat.call("lsb_norm_rows", ws.xh, self.Hp, ws.resid, self.Hp, rows, row0, nw, nb, alpha, n, self.cfg.hidden, self.cfg.rms_eps, kind, int(self.f32))
        self.head(ws.logits, ws.xh, n)
        if self.cfg.softcap:
            nat.call("lsb_softcap", ws.logits, ws.logits.shape[1], n, self.cfg.vocab, self.cfg.softcap)


class _Meta:
    """Columns of a mixer's projections in the projection buffer (-1: it has none) and the padded ranks of its low-rank gates."""

    def __init__(self, offs: List[int], ra: int = 0, rg: int = 0):
        self.offs, self.ra, self.rg = offs, ra, rg

    def shift(self, n: int):
        self.offs = [o + n if o >= 0 else o for o in self.offs]


def _offsets(parts) -> List[int]:
    """Rows at which stacked projections start, each padded to a multiple of 8."""
    offs, o = [], 0
    for t in parts:
        offs.append(o)
        o += _align(t.shape[0], 8)
    return offs


def model_class(cfg: ModelConfig):
    """The device model class of a configuration."""
    from .device_model import DeviceModel
    return BlockModel if cfg.blocks else DeviceModel
