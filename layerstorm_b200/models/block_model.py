"""Models described layer by layer (``ModelConfig.blocks``) on the device: every layer is a mixer (grouped-query attention or a gated delta
rule) and an optional routed feed-forward, each with its own sizes, around a post-norm fp32 residual stream

    x <- x + norm1(mixer(x)),    x <- x + norm2(ffn(x)),    logits = head(norm(x)) * logit_scale.

Same engine, caches and step protocol as :class:`DeviceModel`: attention layers keep a paged cache (one row of all heads' keys and values per
token), delta-rule layers an fp32 state and convolution history per sequence slot.  Steps are any mixture of prompt portions and single tokens.

Two precisions.  ``bfloat16``: weights, activations and the cache in bf16, products accumulated in fp32; the residual stream, norms, routing,
attention scores and weights and the whole recurrence in fp32.  ``float32``: everything in fp32 (FMA units, no reduced-precision products).

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


def block_weight_shapes(cfg: ModelConfig, ranks: Optional[Dict[int, tuple]] = None) -> Dict[str, tuple]:
    """Canonical tensor names and shapes.  ``ranks``: {layer: (decay rank, gate rank)} of delta-rule layers (default: the key head width)."""
    H, out = cfg.hidden, {}
    norm = lambda p: out.update({p + ".weight": (H,)} | ({p + ".bias": (H,)} if cfg.norm_kind == "layer" else {}))
    out["embed.weight"] = out["head.weight"] = (cfg.vocab, H)
    norm("final_norm")
    for i, b in enumerate(cfg.blocks):
        p = f"layers.{i}."
        norm(p + "mix_norm")
        if b.recurrent:
            k, kw, vw = p + "kda.", b.kv_heads * b.dim, b.heads * b.vdim
            ra, rg = (ranks or {}).get(i, (b.dim, b.dim))
            out.update({k + "q": (kw, H), k + "k": (kw, H), k + "v": (vw, H), k + "beta": (b.heads, H), k + "f_a": (ra, H), k + "g_a": (rg, H),
                        k + "f_b": (b.heads * b.dim, ra), k + "g_b": (vw, rg), k + "conv_q": (kw, b.conv), k + "conv_k": (kw, b.conv), k + "conv_v": (vw, b.conv),
                        k + "a_log": (b.heads,), k + "dt_bias": (b.heads * b.dim,), k + "o_norm": (b.vdim,), k + "o": (H, vw)})
        else:
            a, qw, kw, vw = p + "attn.", b.heads * b.dim, b.kv_heads * b.dim, b.kv_heads * b.vdim
            out.update({a + "q": (qw, H), a + "k": (kw, H), a + "v": (vw, H), a + "o": (H, b.heads * b.vdim)})
            if b.qk_norm:
                out.update({a + "q_norm": (qw,), a + "k_norm": (kw,)})
            if b.out_gate:
                out[a + "g"] = (b.heads * b.vdim, H)
            if b.v_mix:
                out[a + "v_mix"] = ()
        if b.experts:
            norm(p + "ffn_norm")
            m = p + "moe."
            out[m + "router"], out[m + "router_bias"] = (b.experts + b.identity, H), (b.experts + b.identity,)
            for e in range(b.experts):
                out.update({m + f"experts.{e}.gate": (b.ff, H), m + f"experts.{e}.up": (b.ff, H), m + f"experts.{e}.down": (H, b.ff)})
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
    if leaf == "weight":                                     # embedding, head
        return t.normal_(0.0, 1.0 if name.startswith("embed") else 0.5 / shape[1] ** 0.5, generator=gen)
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
        att = [b for b in m.cfg.blocks if not b.recurrent]
        if att:
            self.q = z(R * max(b.heads * m.head_pad(b.dim) for b in att), dtype=act)
            self.v_first = z(R, max([b.kv_heads * b.vdim for b in att if b.v_mix], default=1))
            # key splits of the few-row attention: about two blocks per SM, no split shorter than 64 visible keys
            self.splits = {}
            for i, b in enumerate(m.cfg.blocks):
                if not b.recurrent:
                    seen = min(b.window or max_ctx, max_ctx)
                    blocks = R * b.kv_heads * ((b.heads // b.kv_heads + 15) // 16)
                    self.splits[i] = 1 if (m.f32 or R > 64) else max(1, min(32, 296 // blocks, (seen + 63) // 64))
            ns = [(b.heads * self.splits[i], m.head_pad(b.vdim)) for i, b in enumerate(m.cfg.blocks) if not b.recurrent and self.splits[i] > 1]
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
        self.max_mix = 8
        mixing = [i for i, b in enumerate(cfg.blocks) if b.v_mix and not b.recurrent]
        self.v_first_layer = mixing[0] if mixing else -1
        if len({cfg.blocks[i].kv_heads * cfg.blocks[i].vdim for i in mixing}) > 1:
            raise ValueError("layers that mix values must have the same number of value channels")
        for i, b in enumerate(cfg.blocks):
            if b.heads % max(b.kv_heads, 1) or min(b.heads, b.kv_heads, b.dim, b.vdim) < 1:
                raise ValueError(f"layer {i}: {b.heads} heads over {b.kv_heads} groups of widths {b.dim} / {b.vdim}")
            if b.recurrent and b.dim > 256:
                raise ValueError(f"layer {i}: key heads of up to 256 channels, not {b.dim}")
            if b.experts and (b.top > min(32, b.experts + b.identity) or (b.experts + b.identity) % b.groups or b.groups > 64):
                raise ValueError(f"layer {i}: router with {b.experts} + {b.identity} outputs, top {b.top}, {b.groups} groups")

    @staticmethod
    def head_pad(d: int) -> int:
        return int(nat.call("lsb_attn_head_pad", d))

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

        def norm(p, scale=1.0):
            b = p + ".bias"
            return m._vec(w[p + ".weight"]) * scale, (m._vec(w[b]) * scale if b in w else None)

        e = torch.zeros(cfg.vocab, Hp, dtype=torch.bfloat16, device=dev)
        e[:, :H] = w["embed.weight"].to(dev)
        m.embed = e
        hw = w["head.weight"].to(dev)
        m.head = m._mat(hw, cols=Hp)
        m.head.N = cfg.vocab                                   # padding rows of the matrix are never computed
        m.final_norm, m.final_bias = norm("final_norm", cfg.logit_scale)      # the scale of the logits rides on the last norm
        for i, b in enumerate(cfg.blocks):
            p = f"layers.{i}."
            L: dict = {"norm1": norm(p + "mix_norm")}
            if b.recurrent:
                k = p + "kda."
                fb, gb = w[k + "f_b"].to(dev), w[k + "g_b"].to(dev)
                ra, rg = _align(fb.shape[1], 8), _align(gb.shape[1], 8)
                kw, vw = b.kv_heads * b.dim, b.heads * b.vdim
                parts = [w[k + n].to(dev) for n in ("q", "k", "v", "beta", "f_a", "g_a")]
                L["in"] = m._mat(*parts, cols=Hp)
                offs, o = [], 0
                for t in parts:
                    offs.append(o)
                    o += _align(t.shape[0], 8)
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
                L["out"].N = Hp
            else:
                a = p + "attn."
                parts = [w[a + n].to(dev) for n in ("q", "k", "v")] + ([w[a + "g"].to(dev)] if b.out_gate else [])
                L["in"] = m._mat(*parts, cols=Hp)
                offs, o = [], 0
                for t in parts:
                    offs.append(o)
                    o += _align(t.shape[0], 8)
                L["meta"] = _Meta(offs=offs + ([] if b.out_gate else [-1]))
                if b.qk_norm:
                    L["q_norm"], L["k_norm"] = m._vec(w[a + "q_norm"]), m._vec(w[a + "k_norm"])
                if b.alibi:
                    L["slope"] = torch.tensor([2.0 ** (-8.0 * (h + 1) / b.heads) for h in range(b.heads)], dtype=torch.float32, device=dev)
                if b.v_mix:
                    L["v_mix"] = m._vec(w[a + "v_mix"])
                L["out"] = m._mat(w[a + "o"].to(dev), cols=_align(b.heads * b.vdim, 8))
            m.max_proj = max(m.max_proj, L["in"].N)
            m.max_mix = max(m.max_mix, L["out"].K)
            if b.experts:
                mo = p + "moe."
                L["norm2"] = norm(p + "ffn_norm")
                L["router"] = m._mat(w[mo + "router"].to(dev), cols=Hp)        # values of the file's type: fp32-accumulated products are exact in them
                L["router"].N = b.experts + b.identity
                L["router_bias"] = m._vec(w[mo + "router_bias"]) if (mo + "router_bias") in w else None
                # expert width padded to the tensor-core tile where the residual width allows that path
                F = _align(b.ff, 128) if Hp % 128 == 0 else _align(b.ff, 8)
                arena = ExpertArena(expert_layout(m.w_fmt, Hp, F), b.experts, b.experts, dev)
                for x in range(b.experts):
                    g, u, d = (torch.zeros(n, k, dtype=m.act_dtype, device=dev) for n, k in ((F, Hp), (F, Hp), (Hp, F)))
                    g[: b.ff, :H], u[: b.ff, :H], d[:H, : b.ff] = (w[mo + f"experts.{x}.{n}"].to(dev) for n in ("gate", "up", "down"))
                    arena.write_expert(x, QLinear(m.w_fmt, F, Hp, g), QLinear(m.w_fmt, F, Hp, u), QLinear(m.w_fmt, Hp, F, d))
                    arena.slot_of[x] = x
                L["arena"] = arena
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
            else:
                self.kv_cache[i] = z(num_pages, self.page, b.kv_heads * (self.head_pad(b.dim) + self.head_pad(b.vdim)), dtype=self.act_dtype)

    def cache_bytes_per_token(self) -> int:
        return sum(b.kv_heads * (self.head_pad(b.dim) + self.head_pad(b.vdim)) * (4 if self.f32 else 2) for b in self.cfg.blocks if not b.recurrent)

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

    def _moe(self, i: int, b: BlockSpec, L: dict, ws: BlockWorkspace, R: int) -> MoeBuffers:
        mb = ws.moe[self.moe_key(i)]
        n = b.experts + b.identity
        L["router"](mb.logits_r, ws.x, R, ldo=n)
        nat.call("lsb_router_topk_grouped", mb.logits_r, L["router_bias"], mb.ids, mb.wts, R, n, b.top, b.groups, b.keep, 1, int(self.cfg.norm_topk_prob),
                 self.cfg.routed_scale, 0, n, 1)
        self.moe_prepare(L["arena"], mb, ws.x, R, b.experts)
        self.moe_experts(L["arena"], mb, ws.x, R, b.experts, self.cfg.swiglu_limit, mb.miss)
        return mb

    def set_layer_skip(self, skip=(), probe: bool = False):
        if probe:
            raise NotImplementedError("layer-input similarity probing is built for the MLA family")
        super().set_layer_skip([l for l in skip if int(l) != self.v_first_layer], False)

    def forward(self, ws: BlockWorkspace, R: int, nseq: int, logit_row0: int, n_logit_rows: int):
        """One step over the first ``R`` staged rows; logits of rows [logit_row0, logit_row0 + n_logit_rows)."""
        cfg, H, Hp, f32 = self.cfg, self.cfg.hidden, self.Hp, int(self.f32)
        layer = int(cfg.norm_kind == "layer")
        nat.call("lsb_embedding", ws.resid, None if f32 else ws.x, self.embed, ws.tok, R, Hp, 0, cfg.vocab)
        if f32:
            ws.x[:R].copy_(ws.resid[:R])
        for i, (b, L) in enumerate(zip(cfg.blocks, self.layers)):
            if self.aux_capture is not None:
                self._capture_aux(i, ws, R)
            if i in self.skip_layers:
                continue
            (self._delta if b.recurrent else self._attention)(i, b, L, ws, R, nseq)
            L["out"](ws.sub, ws.mix, R, ldo=Hp)
            nw, nb = L["norm1"]
            nat.call("lsb_post_norm", ws.x, Hp, ws.resid, Hp, ws.sub, Hp, nw, nb, R, H, cfg.rms_eps, layer, None, None, None, None, 0, 0, 0, f32)
            if b.experts:
                mb = self._moe(i, b, L, ws, R)
                nw, nb = L["norm2"]
                nat.call("lsb_post_norm", ws.x, Hp, ws.resid, Hp, None, 0, nw, nb, R, H, cfg.rms_eps, layer, mb.y, mb.wts, mb.ids, L["arena"].slot_of, b.top,
                         b.experts, L["arena"].ef.H, f32)
            if self.drift is not None:
                self.drift[f"layer{i:03d}.resid"] = ws.resid[:R, :H].float().cpu()
        if self.aux_capture is not None:
            self._capture_aux(cfg.n_layers, ws, R)
        if n_logit_rows:
            self.emit_logits(ws, logit_row0, n_logit_rows)

    def emit_logits(self, ws: BlockWorkspace, row0: int, n: int, rows: Optional[torch.Tensor] = None):
        """Logits of step rows [row0, row0 + n), or of the ``n`` rows listed in ``rows`` (int32, device), after :meth:`forward`."""
        nat.call("lsb_norm_rows", ws.xh, self.Hp, ws.resid, self.Hp, rows, row0, self.final_norm, self.final_bias, n, self.cfg.hidden, self.cfg.rms_eps,
                 int(self.cfg.norm_kind == "layer"), int(self.f32))
        self.head(ws.logits, ws.xh, n)


class _Meta:
    """Column offsets of a layer's fused input projection and the padded ranks of its low-rank gates."""

    def __init__(self, offs: List[int], ra: int = 0, rg: int = 0):
        self.offs, self.ra, self.rg = offs, ra, rg


def model_class(cfg: ModelConfig):
    """The device model class of a configuration."""
    from .device_model import DeviceModel
    return BlockModel if cfg.blocks else DeviceModel
