"""Models described layer by layer (``ModelConfig.blocks``) on the device: every layer is a mixer (grouped-query attention, latent attention or
a gated delta rule) and an optional feed-forward (a dense gated unit or routed experts), each with its own sizes, around an fp32 residual stream.
The norms stand on every sublayer's output (``norm_place`` "post") or on both its sides ("sandwich"; n_in is the identity for "post"):

    x <- x + n_out(mixer(n_in(x))),    x <- x + n_out(ffn(n_in(x))),    logits = head(norm(x)) * logit_scale,

and a layer may end with an update from its slice e of a per-token table: x <- x + rms(W_p (gelu(W_g x) * e)).

Same engine, caches and step protocol as :class:`DeviceModel`: attention layers keep a paged cache (one row of all heads' keys and values per
token; latent layers one row for all heads, which later layers may read instead of keeping their own), delta-rule layers an fp32 state and
convolution history per sequence slot.  Steps are any mixture of prompt portions and single tokens.

Two precisions.  ``bfloat16``: weights, activations and the cache in bf16, products accumulated in fp32; the residual stream, norms, routing,
attention scores and weights, rotations and the whole recurrence in fp32.  ``float32``: everything in fp32 (FMA units, no reduced-precision
products).

Sizes are padded where kernels want it: the residual width to a multiple of 8, projection blocks to multiples of 8 rows, head widths and
expert widths to the kernels' tiles; padding holds zeros and never reaches a result.
"""
from __future__ import annotations

import logging
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


def block_weight_shapes(cfg: ModelConfig, ranks: Optional[Dict[int, tuple]] = None) -> Dict[str, tuple]:
    """Canonical tensor names and shapes.  ``ranks``: {layer: (decay rank, gate rank)} of delta-rule layers (default: the key head width)."""
    H, out = cfg.hidden, {}
    extra = {"rms": (), "layer": ("bias",), "tanh": ("bias", "alpha")}[cfg.norm_kind]
    norm = lambda p: out.update({p + ".weight": (H,)} | {f"{p}.{k}": () if k == "alpha" else (H,) for k in extra})
    out["embed.weight"] = out["head.weight"] = (cfg.vocab, H)
    if cfg.side_dim:
        out["side_embed.weight"] = (cfg.vocab, cfg.n_layers * cfg.side_dim)
    norm("final_norm")
    for i, b in enumerate(cfg.blocks):
        p = f"layers.{i}."
        norm(p + "mix_norm")
        if cfg.norm_place == "sandwich":
            norm(p + "mix_post_norm")
        if b.recurrent:
            k, kw, vw = p + "kda.", b.kv_heads * b.dim, b.heads * b.vdim
            ra, rg = (ranks or {}).get(i, (b.dim, b.dim))
            out.update({k + "q": (kw, H), k + "k": (kw, H), k + "v": (vw, H), k + "beta": (b.heads, H), k + "f_a": (ra, H), k + "g_a": (rg, H),
                        k + "f_b": (b.heads * b.dim, ra), k + "g_b": (vw, rg), k + "conv_q": (kw, b.conv), k + "conv_k": (kw, b.conv), k + "conv_v": (vw, b.conv),
                        k + "a_log": (b.heads,), k + "dt_bias": (b.heads * b.dim,), k + "o_norm": (b.vdim,), k + "o": (H, vw)})
        elif b.latent:
            a = p + "attn."
            out.update({a + "q": (b.heads * (b.dim + b.rot_dim), H), a + "k_b": (b.heads * b.dim, b.kv_rank), a + "v_b": (b.heads * b.vdim, b.kv_rank),
                        a + "o": (H, b.heads * b.vdim)})
            if b.kv_from < 0:
                out.update({a + "kv_a": (b.kv_rank + b.rot_dim, H), a + "kv_a_norm": (b.kv_rank,)})
            if b.head_gate:
                out[a + "g"] = (b.heads, H)
        else:
            a, qw, kw, vw = p + "attn.", b.heads * b.dim, b.kv_heads * b.dim, b.kv_heads * b.vdim
            out.update({a + "q": (qw, H), a + "k": (kw, H), a + "v": (vw, H), a + "o": (H, b.heads * b.vdim)})
            if b.qk_norm:
                out.update({a + "q_norm": (qw,), a + "k_norm": (kw,)})
            if b.out_gate:
                out[a + "g"] = (b.heads * b.vdim, H)
            if b.v_mix:
                out[a + "v_mix"] = ()
        if b.has_ff:
            norm(p + "ffn_norm")
            if cfg.norm_place == "sandwich":
                norm(p + "ffn_post_norm")
        glu = lambda m, ff: out.update({m + "gate": (ff, H), m + "up": (ff, H), m + "down": (H, ff)})
        if b.dense_ff:
            glu(p + "mlp.", b.dense_ff)
        if b.experts:
            m = p + "moe."
            out[m + "router"] = (b.experts + b.identity, H)
            if b.correction:
                out[m + "router_bias"] = (b.experts + b.identity,)
            for e in range(b.experts):
                glu(m + f"experts.{e}.", b.ff)
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
    if leaf.startswith("conv_"):
        return t.uniform_(-0.7, 0.7, generator=gen)
    if leaf == "v_mix":
        return t.uniform_(0.2, 0.6, generator=gen)
    if leaf in ("bias", "router_bias"):
        return t.normal_(0.0, 0.1, generator=gen)
    if leaf == "alpha":
        return t.uniform_(0.4, 1.0, generator=gen)
    if leaf == "weight":                                     # token tables, head
        return t.normal_(0.0, 1.0 if "embed" in name else 0.5 / shape[1] ** 0.5, generator=gen)
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
        self.x = z(R, Hp, dtype=act)                 # the residual stream in the activation type: what every sublayer reads
        self.resid = z(R, Hp)
        self.sub = z(R, Hp)
        self.xh = z(n_logit_rows, Hp, dtype=act)
        self.proj = z(R, m.max_proj)
        self.mix = z(R, m.max_mix, dtype=act)        # a mixer's output in front of its output projection
        lat = [b for b in m.cfg.blocks if b.latent]
        att = [b for b in m.cfg.blocks if not b.recurrent and not b.latent]
        if lat:
            self.q_lat = z(R * max(b.heads * m.latent_row(b) for b in lat), dtype=act)
            self.q_nope = z(R * max(b.heads * _align(b.dim, 8) for b in lat), dtype=torch.bfloat16) if not m.f32 and R >= 8 else None
            self.o_lat = z(R * max(b.heads * m.latent_pad(b.kv_rank) for b in lat), dtype=act)
            self.lat_splits = {i: 1 if R > 64 else int(nat.call("lsb_latent_splits", R, b.heads, b.kv_rank, b.rot_dim, max_ctx, int(m.f32)))
                               for i, b in enumerate(m.cfg.blocks) if b.latent}
            self.lat_parts = {i: int(nat.call("lsb_latent_partials", n)) for i, n in self.lat_splits.items()}
            ns = [(b.heads * self.lat_parts[i], m.latent_pad(b.kv_rank)) for i, b in enumerate(m.cfg.blocks) if self.lat_parts.get(i, 1) > 1]
            self.lat_o_part = z(R * max((n * w for n, w in ns), default=1))
            self.lat_ml_part = z(2 * R * max((n for n, _ in ns), default=1))
        dense = max((_align(max(b.dense_ff, b.shared_ff), 8) for b in m.cfg.blocks), default=0)
        self.glu = z(R * dense, dtype=act) if dense else None
        self.side = z(R, _align(m.cfg.side_dim, 8), dtype=act) if m.cfg.side_dim else None
        if att:
            self.q = z(R * max(b.heads * m.head_pad(b.dim) for b in att), dtype=act)
            self.v_first = z(R, max([b.kv_heads * b.vdim for b in att if b.v_mix], default=1))
            # key splits of the few-row attention: about two blocks per SM, no split shorter than 64 visible keys
            self.splits = {}
            for i, b in enumerate(m.cfg.blocks):
                if not b.recurrent and not b.latent:
                    seen = min(b.window or max_ctx, max_ctx)
                    blocks = R * b.kv_heads * ((b.heads // b.kv_heads + 15) // 16)
                    self.splits[i] = 1 if (m.f32 or R > 64) else max(1, min(32, 296 // blocks, (seen + 63) // 64))
            ns = [(b.heads * self.splits[i], m.head_pad(b.vdim)) for i, b in enumerate(m.cfg.blocks) if self.splits.get(i, 1) > 1]
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
        self._delta = self._chunk = None

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
        for i, b in enumerate(cfg.blocks):
            if b.heads % max(b.kv_heads, 1) or min(b.heads, b.kv_heads, b.dim, b.vdim) < 1:
                raise ValueError(f"layer {i}: {b.heads} heads over {b.kv_heads} groups of widths {b.dim} / {b.vdim}")
            if b.latent and (b.kv_rank < 1 or b.rot_dim < 2 or b.rot_dim % 2):
                raise ValueError(f"layer {i}: latent rows of {b.kv_rank} + {b.rot_dim} channels")
            if b.recurrent and b.dim > 256:
                raise ValueError(f"layer {i}: key heads of up to 256 channels, not {b.dim}")
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
            return kind, m._vec(w[p + ".weight"]) * scale, (m._vec(w[b]) * scale if b in w else None), (m._vec(w[al]) if al in w else None)

        def stacked(parts, cols=Hp):
            """The parts as one projection and the row at which each starts."""
            offs, o = [], 0
            for t in parts:
                offs.append(o)
                o += _align(t.shape[0], 8)
            return m._mat(*parts, cols=cols), offs

        e = torch.zeros(cfg.vocab, Hp, dtype=torch.bfloat16, device=dev)
        e[:, :H] = w["embed.weight"].to(dev)
        m.embed = e
        hw = w["head.weight"].to(dev)
        m.head = m._mat(hw, cols=Hp)
        m.head.N = cfg.vocab                                   # padding rows of the matrix are never computed
        m.final_norm = norm("final_norm", cfg.logit_scale)     # the scale of the logits rides on the last norm
        if cfg.side_dim:
            m.side_embed = w["side_embed.weight"].to(dev).to(torch.bfloat16).contiguous()
        for i, b in enumerate(cfg.blocks):
            p = f"layers.{i}."
            L: dict = {"mix_in": norm(p + "mix_norm"), "mix_out": norm(p + "mix_post_norm")} if sandwich else {"mix_in": NO_NORM, "mix_out": norm(p + "mix_norm")}
            if b.recurrent:
                k = p + "kda."
                fb, gb = w[k + "f_b"].to(dev), w[k + "g_b"].to(dev)
                ra, rg = _align(fb.shape[1], 8), _align(gb.shape[1], 8)
                kw, vw = b.kv_heads * b.dim, b.heads * b.vdim
                parts = [w[k + n].to(dev) for n in ("q", "k", "v", "beta", "f_a", "g_a")]
                L["in"], offs = stacked(parts)
                L["meta"] = _Meta(offs=offs, ra=ra, rg=rg)
                pad = lambda t, n: torch.nn.functional.pad(t.float(), (0, n - t.shape[1])).to(m.act_dtype).contiguous()
                L["w_a"], L["w_g"] = pad(fb, ra), pad(gb, rg)
                if not m.f32:
                    # [W | W]: many rows take the low-rank products on the tensor cores with (hi | lo) activations
                    L["w_a2"], L["w_g2"] = torch.cat([L["w_a"]] * 2, 1).contiguous(), torch.cat([L["w_g"]] * 2, 1).contiguous()
                for n in ("conv_q", "conv_k", "conv_v"):
                    t = w[k + n].to(dev).float().contiguous()
                    if tuple(t.shape) != ((vw if n == "conv_v" else kw), b.conv):
                        raise ValueError(f"{k + n}: shape {tuple(t.shape)}")
                    L[n] = t
                L["a_exp"], L["dt_bias"], L["o_norm"] = torch.exp(m._vec(w[k + "a_log"])), m._vec(w[k + "dt_bias"]), m._vec(w[k + "o_norm"])
                L["out"] = m._mat(w[k + "o"].to(dev), cols=_align(vw, 8))
            elif b.latent:
                a, own = p + "attn.", b.kv_from < 0
                names = ["q"] + (["kv_a"] if own else []) + (["g"] if b.head_gate else [])
                L["in"], offs = stacked([w[a + n].to(dev) for n in names])
                at = dict(zip(names, offs))
                L["meta"] = _Meta(offs=[at["q"], at.get("kv_a", -1), at.get("g", -1)])
                dnp, dlp = _align(b.dim, 8), m.latent_pad(b.kv_rank)
                uk, uv = w[a + "k_b"].to(dev).view(b.heads, b.dim, b.kv_rank), w[a + "v_b"].to(dev).view(b.heads, b.vdim, b.kv_rank)
                L["w_uk"] = torch.zeros(b.heads, dlp, dnp, dtype=m.act_dtype, device=dev)
                L["w_uk"][:, : b.kv_rank, : b.dim] = uk.transpose(1, 2)
                L["w_uv"] = torch.zeros(b.heads, b.vdim, dlp, dtype=m.act_dtype, device=dev)
                L["w_uv"][:, :, : b.kv_rank] = uv
                if not m.f32:
                    # the same two, one after the other per position: what long prompt runs make keys and values with
                    dnw, dvp = _align(b.dim, 16), m.head_pad(b.vdim)
                    L["w_kv"] = torch.zeros(b.heads * (dnw + dvp), dlp, dtype=m.act_dtype, device=dev)
                    L["w_kv"][: b.heads * dnw].view(b.heads, dnw, dlp)[:, : b.dim, : b.kv_rank] = uk
                    L["w_kv"][b.heads * dnw:].view(b.heads, dvp, dlp)[:, : b.vdim, : b.kv_rank] = uv
                if own:
                    L["kv_norm"] = m._vec(w[a + "kv_a_norm"])
                L["inv_freq"] = torch.tensor([b.rot_base ** (-2.0 * j / b.rot_dim) for j in range(b.rot_dim // 2)], dtype=torch.float64, device=dev)
                L["out"] = m._mat(w[a + "o"].to(dev), cols=_align(b.heads * b.vdim, 8))
            else:
                a = p + "attn."
                parts = [w[a + n].to(dev) for n in ("q", "k", "v")] + ([w[a + "g"].to(dev)] if b.out_gate else [])
                L["in"], offs = stacked(parts)
                L["meta"] = _Meta(offs=offs + ([] if b.out_gate else [-1]))
                if b.qk_norm:
                    L["q_norm"], L["k_norm"] = m._vec(w[a + "q_norm"]), m._vec(w[a + "k_norm"])
                if b.alibi:
                    L["slope"] = torch.tensor([2.0 ** (-8.0 * (h + 1) / b.heads) for h in range(b.heads)], dtype=torch.float32, device=dev)
                if b.v_mix:
                    L["v_mix"] = m._vec(w[a + "v_mix"])
                L["out"] = m._mat(w[a + "o"].to(dev), cols=_align(b.heads * b.vdim, 8))
            L["out"].N = Hp
            m.max_proj = max(m.max_proj, L["in"].N)
            m.max_mix = max(m.max_mix, L["out"].K)
            if b.has_ff:
                L["ff_in"], L["ff_out"] = (norm(p + "ffn_norm"), norm(p + "ffn_post_norm")) if sandwich else (NO_NORM, norm(p + "ffn_norm"))
            if b.dense_ff:
                L["ff"], L["ff_offs"] = stacked([w[p + f"mlp.{n}"].to(dev) for n in ("gate", "up")])
                L["ff_down"] = m._mat(w[p + "mlp.down"].to(dev))
                L["ff_down"].N = Hp
                m.max_proj = max(m.max_proj, L["ff"].N)
            if b.experts:
                mo = p + "moe."
                # the router and - where there is one - the shared expert's gate, up and output-gate rows are one product (values of the file's
                # type: fp32-accumulated products are exact in them)
                parts = [w[mo + "router"].to(dev)] + ([w[mo + n].to(dev) for n in ("shared.0.gate", "shared.0.up", "shared_gate")] if b.shared_ff else [])
                L["router"], L["ff_offs"] = stacked(parts)
                L["router_bias"] = m._vec(w[mo + "router_bias"]) if b.correction and (mo + "router_bias") in w else None
                if b.shared_ff:
                    L["ff_down"] = m._mat(w[mo + "shared.0.down"].to(dev))
                    L["ff_down"].N = Hp
                m.max_proj = max(m.max_proj, L["router"].N)
                # expert width padded to the tensor-core tile where the residual width allows that path
                F = _align(b.ff, 128) if Hp % 128 == 0 else _align(b.ff, 8)
                arena = ExpertArena(expert_layout(m.w_fmt, Hp, F), b.experts, b.experts, dev)
                for x in range(b.experts):
                    g, u, d = (torch.zeros(n, k, dtype=m.act_dtype, device=dev) for n, k in ((F, Hp), (F, Hp), (Hp, F)))
                    g[: b.ff, :H], u[: b.ff, :H], d[:H, : b.ff] = (w[mo + f"experts.{x}.{n}"].to(dev) for n in ("gate", "up", "down"))
                    arena.write_expert(x, QLinear(m.w_fmt, F, Hp, g), QLinear(m.w_fmt, F, Hp, u), QLinear(m.w_fmt, Hp, F, d))
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
        for i, b in enumerate(self.cfg.blocks):
            if b.recurrent:
                self.kda_state[i] = z(n_slots, b.heads, b.vdim, int(nat.call("lsb_delta_key_pad", b.dim)))
                self.kda_conv[i] = z(n_slots, b.heads, 2 * b.dim + b.vdim, b.conv - 1)
            elif b.latent:
                if b.kv_from < 0:
                    self.kv_cache[i] = z(num_pages, self.page, self.latent_row(b), dtype=self.act_dtype)
            else:
                self.kv_cache[i] = z(num_pages, self.page, b.kv_heads * (self.head_pad(b.dim) + self.head_pad(b.vdim)), dtype=self.act_dtype)

    def cache_bytes_per_token(self) -> int:
        width = lambda b: ((self.latent_row(b) if b.kv_from < 0 else 0) if b.latent else b.kv_heads * (self.head_pad(b.dim) + self.head_pad(b.vdim)))
        return sum(width(b) * (4 if self.f32 else 2) for b in self.cfg.blocks if not b.recurrent)

    # ------------------------------------------------------------------ forward
    def _resid_rows(self, ws, R: int, H: int) -> torch.Tensor:
        return ws.resid[:R, :H]

    def _attention(self, i: int, b: BlockSpec, L: dict, ws: BlockWorkspace, R: int, nseq: int):
        dkp, dvp, ldp = self.head_pad(b.dim), self.head_pad(b.vdim), self.max_proj
        oq, ok, ov, og = L["meta"].offs
        L["in"](ws.proj, ws.x, R, ldo=ldp)
        mix = 0 if not b.v_mix else (1 if i == self.v_first_layer else 2)
        nat.call("lsb_attn_prep", ws.proj, ldp, oq, ok, ov, L.get("q_norm"), L.get("k_norm"), self.cfg.rms_eps, ws.v_first if mix else None, mix,
                 L.get("v_mix"), ws.q, self.kv_cache[i], self.block_table, self.max_pages, ws.row_seq, ws.row_pos, R, b.heads, b.kv_heads, b.dim, b.vdim,
                 dkp, dvp, self.page, int(self.f32))
        nat.call("lsb_attn", ws.q, self.kv_cache[i], self.block_table, self.max_pages, self.page, ws.row_seq, ws.row_pos, ws.seq_row0, ws.seq_nrows, nseq,
                 max(ws.seq_rows), ws.proj, ldp, og, ws.mix, L["out"].K, ws.o_part, ws.ml_part, ws.splits[i], R, b.heads, b.kv_heads, b.dim, b.vdim, dkp, dvp,
                 b.window, b.scale, L.get("slope"), int(self.f32))

    def _latent(self, i: int, b: BlockSpec, L: dict, ws: BlockWorkspace, R: int, nseq: int):
        cache = self.kv_cache[i if b.kv_from < 0 else b.kv_from]
        L["in"](ws.proj, ws.x, R, ldo=self.max_proj)
        # long runs one by one, what lies between them together
        rows, row0, j = ws.seq_rows, 0, 0
        while j < nseq:
            k, n = j + 1, rows[j]
            if self._expands(b, rows[j], ws.seq_end[j]):
                self._latent_run(b, L, ws, cache, row0, n, j)
            else:
                while k < nseq and not self._expands(b, rows[k], ws.seq_end[k]):
                    n, k = n + rows[k], k + 1
                self._latent_rows(i, b, L, ws, cache, row0, n, j, k)
            row0, j = row0 + n, k

    def _latent_rows(self, i: int, b: BlockSpec, L: dict, ws: BlockWorkspace, cache, r0: int, R: int, j: int, k: int):
        """Step rows [r0, r0 + R) (sequences j .. k - 1 of the step) in the latent space."""
        oq, okv, og = L["meta"].offs
        H, ld, K, f32, err = b.heads, self.max_proj, L["out"].K, int(self.f32), TcScratch.get(self.device).err
        q, o_lat, proj, seq, pos = ws.q_lat[r0 * H * self.latent_row(b):], ws.o_lat[r0 * H * L["w_uv"].shape[2]:], ws.proj[r0:], ws.row_seq[r0:], ws.row_pos[r0:]
        nat.call("lsb_latent_query", proj, ld, oq, okv, L.get("kv_norm"), self.cfg.rms_eps, L["inv_freq"], L["w_uk"], q, ws.q_nope, cache, self.block_table,
                 self.max_pages, self.page, seq, pos, R, H, b.dim, L["w_uk"].shape[2], b.rot_dim, b.kv_rank, f32, err)
        # seq_row0 holds row numbers of the step, so runs get the whole buffers (steps with key splits have no long runs: r0 is 0)
        run = max(ws.seq_rows[j:k])
        rows = (q, proj, seq, pos, o_lat) if run == 1 else (ws.q_lat, ws.proj, ws.row_seq, ws.row_pos, ws.o_lat)
        nat.call("lsb_latent_attn", rows[0], cache, self.block_table, self.max_pages, self.page, rows[2], rows[3], ws.seq_row0[j:], ws.seq_nrows[j:], k - j, run,
                 rows[1], ld, og, rows[4], ws.lat_o_part, ws.lat_ml_part, ws.lat_splits[i], R, H, b.kv_rank, b.rot_dim, b.scale, f32)
        nat.call("lsb_latent_out", ws.mix.view(-1)[r0 * K:], K, o_lat, ws.lat_o_part, ws.lat_ml_part, ws.lat_parts[i], L["w_uv"], proj, ld, og, seq, R, H, b.kv_rank,
                 b.vdim, f32, err)

    def _latent_run(self, b: BlockSpec, L: dict, ws: BlockWorkspace, cache, r0: int, R: int, j: int):
        """Step rows [r0, r0 + R), a run of sequence j, over keys and values of every head, made for this step from the cached rows."""
        oq, okv, og = L["meta"].offs
        H, ld, K, err, T = b.heads, self.max_proj, L["out"].K, TcScratch.get(self.device).err, ws.seq_end[j]
        dnw, dvp, drp = _align(b.dim, 16), self.head_pad(b.vdim), self.latent_pad(b.rot_dim)
        Tm, proj, seq, pos = _align(T, 256), ws.proj[r0:], ws.row_seq[r0:], ws.row_pos[r0:]
        q, lat, kv = self._expand_scratch(ws.R, R * H * (dnw + drp), Tm * self.latent_pad(b.kv_rank), Tm * (H * (dnw + dvp) + drp))
        nat.call("lsb_latent_expand", proj, ld, oq, okv, L.get("kv_norm"), self.cfg.rms_eps, L["inv_freq"], L["w_kv"], q, lat, kv, cache, self.block_table,
                 self.max_pages, self.page, seq, pos, R, T, Tm, H, b.dim, dnw, b.rot_dim, b.kv_rank, dvp, err)
        nat.call("lsb_attn_run", q, kv, Tm, self.zero, seq, pos, self.zero, ws.seq_nrows[j:], proj, ld, og, ws.mix.view(-1)[r0 * K:], K, R, H, dnw, drp, b.vdim, dvp,
                 b.scale)

    def _expands(self, b: BlockSpec, R: int, T: int) -> bool:
        """Whether a run of R rows over T positions is worth writing keys and values out for (and the kernels take the sizes): fewer operations per
        (query, key), against a product over all positions that runs about four times as fast per operation."""
        dnw, dvp = _align(b.dim, 16), self.head_pad(b.vdim)
        row = b.heads * (dnw + dvp) + self.latent_pad(b.rot_dim)
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

    def _delta(self, i: int, b: BlockSpec, L: dict, ws: BlockWorkspace, R: int, nseq: int):
        mt = L["meta"]
        L["in"](ws.proj, ws.x, R, ldo=self.max_proj)
        rows = ws.seq_rows
        few = max(rows) <= FEW_ROWS and b.vdim <= nat.call("lsb_delta_few_max_dv", b.dim)
        scratch = chunk_ws = None
        long_, chunks = [], 0
        if not few:
            long_ = [n for n in rows if n >= LONG_ROWS] if b.dim <= 128 else []
            chunks = sum((n + 63) // 64 for n in long_)
            scratch, chunk_ws = ws.delta_scratch(b, R, mt.ra, mt.rg, chunks)
        oq, ok, ov, ob, oa, og = mt.offs
        nat.call("lsb_delta_forward", ws.proj, self.max_proj, oq, ok, ov, ob, oa, og, mt.ra, mt.rg, L["w_a"], L["w_g"], L.get("w_a2"), L.get("w_g2"),
                 L["conv_q"], L["conv_k"], L["conv_v"], L["a_exp"], L["dt_bias"], L["o_norm"], self.kda_state[i], self.kda_conv[i], ws.seq_row0,
                 ws.seq_nrows, ws.seq_slot, ws.mix, L["out"].K, nseq, R, b.heads, b.kv_heads, b.dim, b.vdim, b.conv, 0 if b.decay == "softplus" else 1,
                 b.dim ** -0.5, b.decay_bound, self.cfg.rms_eps, int(self.f32), int(few), scratch, len(rows) - len(long_), len(long_), chunks, LONG_ROWS,
                 chunk_ws, TcScratch.get(self.device).err)

    def _glu(self, L: dict, ws: BlockWorkspace, R: int, ff: int, offs, limit=0.0, alpha=1.0, shift=0.0):
        """Gated unit over columns of the projection in ``ws.proj`` and its down product into ``ws.sub``; ``offs``: gate, up, output gate (-1: none)."""
        K = L["ff_down"].K
        nat.call("lsb_glu", ws.glu, K, ws.proj, self.max_proj, *offs, R, ff, limit, alpha, shift, int(self.f32))
        L["ff_down"](ws.sub, ws.glu, R, ldo=self.Hp)

    def _moe(self, i: int, b: BlockSpec, L: dict, ws: BlockWorkspace, R: int) -> MoeBuffers:
        mb, cfg = ws.moe[self.moe_key(i)], self.cfg
        n = b.experts + b.identity
        L["router"](ws.proj, ws.x, R, ldo=self.max_proj)
        nat.call("lsb_router_topk_grouped", ws.proj, L["router_bias"], mb.ids, mb.wts, R, n, b.top, b.groups, b.keep, {"sigmoid": 0, "softmax": 1}[b.scoring],
                 int(cfg.norm_topk_prob), cfg.routed_scale, 0, self.max_proj, 1)
        if b.shared_ff:
            self._glu(L, ws, R, b.shared_ff, L["ff_offs"][1:], b.shared_limit, b.act_alpha, b.act_shift)
        self.moe_prepare(L["arena"], mb, ws.x, R, b.experts)
        plain = b.act_alpha == 1.0 and b.act_shift == 0.0 and not b.scale_input
        act = None if plain else (b.act_alpha, b.act_shift, mb.wts if b.scale_input else None)
        self.moe_experts(L["arena"], mb, ws.x, R, b.experts, b.limit, mb.miss, act)
        return mb

    def _update(self, ws: BlockWorkspace, R: int, post: tuple, pre: tuple, sub=None, mb: Optional[MoeBuffers] = None, b: Optional[BlockSpec] = None,
                L: Optional[dict] = None):
        """resid += post(sub + expert sum), x = pre(resid)."""
        Hp, y = self.Hp, (None, None, None, None, 0, 0, 0)
        if mb is not None:
            y = (mb.y, None if b.scale_input else mb.wts, mb.ids, L["arena"].slot_of, b.top, b.experts, L["arena"].ef.H)
        nat.call("lsb_resid_update", ws.x, Hp, ws.resid, Hp, sub, Hp, *post, *pre, R, self.cfg.hidden, self.cfg.rms_eps, *y, int(self.f32))

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
        super().set_layer_skip([l for l in skip if int(l) not in keep], False)

    def forward(self, ws: BlockWorkspace, R: int, nseq: int, logit_row0: int, n_logit_rows: int):
        """One step over the first ``R`` staged rows; logits of rows [logit_row0, logit_row0 + n_logit_rows)."""
        cfg, H, Hp, f32 = self.cfg, self.cfg.hidden, self.Hp, int(self.f32)
        run = [i for i in range(cfg.n_layers) if i not in self.skip_layers]
        enters = dict(zip([-1] + run, [self.layers[i]["mix_in"] for i in run] + [NO_NORM]))       # norm in front of the layer that follows
        plain = enters[-1] is NO_NORM
        nat.call("lsb_embedding_scaled", ws.resid, ws.x if plain and not f32 else None, self.embed, ws.tok, R, Hp, 0, cfg.vocab, cfg.embed_scale)
        if not plain or f32:
            self._update(ws, R, NO_NORM, enters[-1])
        for i in range(cfg.n_layers):
            if self.aux_capture is not None:
                self._capture_aux(i, ws, R)
            if i not in enters:
                continue
            b, L = cfg.blocks[i], self.layers[i]
            (self._delta if b.recurrent else (self._latent if b.latent else self._attention))(i, b, L, ws, R, nseq)
            L["out"](ws.sub, ws.mix, R, ldo=Hp)
            last = NO_NORM if cfg.side_dim else enters[i]
            self._update(ws, R, L["mix_out"], L["ff_in"] if b.has_ff else last, ws.sub)
            if b.experts:
                mb = self._moe(i, b, L, ws, R)
                self._update(ws, R, L["ff_out"], last, ws.sub if b.shared_ff else None, mb, b, L)
            elif b.dense_ff:
                L["ff"](ws.proj, ws.x, R, ldo=self.max_proj)
                self._glu(L, ws, R, b.dense_ff, (*L["ff_offs"], -1))
                self._update(ws, R, L["ff_out"], last, ws.sub)
            if cfg.side_dim:
                self._side(i, L, ws, R)
                self._update(ws, R, L["side_norm"], enters[i], ws.sub)
            if self.drift is not None:
                self.drift[f"layer{i:03d}.resid"] = ws.resid[:R, :H].float().cpu()
        if self.aux_capture is not None:
            self._capture_aux(cfg.n_layers, ws, R)
        if n_logit_rows:
            self.emit_logits(ws, logit_row0, n_logit_rows)

    def emit_logits(self, ws: BlockWorkspace, row0: int, n: int, rows: Optional[torch.Tensor] = None):
        """Logits of step rows [row0, row0 + n), or of the ``n`` rows listed in ``rows`` (int32, device), after :meth:`forward`."""
        kind, nw, nb, alpha = self.final_norm
        nat.call("lsb_norm_rows", ws.xh, self.Hp, ws.resid, self.Hp, rows, row0, nw, nb, alpha, n, self.cfg.hidden, self.cfg.rms_eps, kind, int(self.f32))
        self.head(ws.logits, ws.xh, n)


class _Meta:
    """Column offsets of a layer's fused input projection and the padded ranks of its low-rank gates."""

    def __init__(self, offs: List[int], ra: int = 0, rg: int = 0):
        self.offs, self.ra, self.rg = offs, ra, rg


def model_class(cfg: ModelConfig):
    """The device model class of a configuration."""
    from .device_model import DeviceModel
    return BlockModel if cfg.blocks else DeviceModel
