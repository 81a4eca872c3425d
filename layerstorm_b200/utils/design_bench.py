"""Prefill and decode throughput of a model design at layer sizes of a real model (random weights), beside the framework's closest other
design at equal size, with the device time of every kernel launcher.

    python bench.py --design gazutar|rubasun|fasodra|nivasun [--design-sizes 2048,4096]

Gazutar's neighbour is a KDA + MLA model of the same width, heads, experts and layer pattern (plain residual stream, dense latent attention),
Rubasun's an MLA + MoE model of the same width, heads, latent rows, experts and shared expert, Fasodra's the Gazutar model of the same width,
attention heads and expert parameters, Nivasun's the Rubasun model (latent attention, gated shared expert) and the Gazutar model (windowed
attention) of the same width, heads and experts.
Per launcher: all its calls of one step, recorded from an eager pass and replayed back to back in a CUDA graph (other layers' operands in
between, so that a layer's weights are not left over in L2), divided by the number of calls.  Fractions are of the measured peaks
(MEASURED_PEAKS.json): bytes or FLOPs that the operation has to move or do, over the launcher's time.
"""
from __future__ import annotations

import json
import os
import statistics

import torch

from ..models.block_model import model_class
from ..models.config import ModelConfig, fasodra_config, gazutar_config, nivasun_config, rubasun_config
from ..ops import _native as nat
from ..runtime.engine import Engine

N_LAYERS, EVERY, TOP = 8, 4, 8


def gazutar_pair(hidden: int):
    """(Gazutar, neighbour) of one size: 128-wide heads, experts of half the width, every fourth layer attention."""
    heads, att_heads, kv, experts, ff, vocab = hidden // 64, hidden // 128, max(1, hidden // 512), hidden // 64, hidden // 2, 65536
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": 8, "top": TOP, "groups": {"count": 8, "keep": 4}}}
    att = {"heads": att_heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 4096}, "v_mix": True}
    dlt = {"heads": heads, "kv_heads": heads, "dim": 128, "vdim": 128, "conv": 4}
    g = gazutar_config({"name": f"gazutar-{hidden}", "vocab": vocab, "width": hidden, "norm": {"eps": 1e-5}, "logit_scale": 0.5, "layers": [
        {"type": "attention", "mixer": att, "mlp": mlp} if i % EVERY == EVERY - 1 else {"type": "channel_delta", "mixer": dlt, "mlp": mlp} for i in range(N_LAYERS)]})
    k = ModelConfig(name=f"kda-mla-{hidden}", architecture="glm5_next", hidden=hidden, n_layers=N_LAYERS, vocab=vocab, rms_eps=1e-5, n_heads=att_heads,
                    q_lora=hidden * 3 // 8, kv_lora=512, qk_nope=128, qk_rope=0, v_head=128, dense_inter=1024, first_k_dense=0, n_routed=experts, top_k=TOP,
                    n_shared=0, moe_inter=ff, scoring="softmax", n_group=8, topk_group=4, norm_topk_prob=False, router_bias=True,
                    layer_types=["mla" if i % EVERY == EVERY - 1 else "kda" for i in range(N_LAYERS)], kda_heads=heads, kda_head_dim=128, kda_rank=128)
    return g, k


def rubasun_pair(hidden: int):
    """(Rubasun, neighbour) of one size: 128 + 64 wide heads over rows of 512 + 64, experts of half the width, a dense first layer; every second
    Rubasun layer reads the rows of the one before it, and every layer takes a per-token input of 256 channels."""
    heads, experts, ff, vocab = hidden // 128, hidden // 64, hidden // 2, 65536
    mixer = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "rot": {"base": 10000.0, "dims": 64}, "scale": 192 ** -0.5}
    moe = {"kind": "moe", "expert": {"ff": ff, "limit": 7.0}, "router": {"experts": experts, "top": TOP}, "shared": {"ff": ff, "limit": 7.0}}
    g = rubasun_config({"name": f"rubasun-{hidden}", "vocab": vocab, "width": hidden, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "token_side": {"dim": 256}, "layers": [
        {"type": "latent_attention", "mixer": mixer | ({"kv_from": i - 1} if i % 2 else {}), "mlp": moe if i else {"kind": "dense", "ff": 3 * hidden}} for i in range(N_LAYERS)]})
    k = ModelConfig(name=f"mla-moe-{hidden}", architecture="deepseek_v3", hidden=hidden, n_layers=N_LAYERS, vocab=vocab, rms_eps=1e-5, n_heads=heads,
                    q_lora=hidden * 3 // 8, kv_lora=512, qk_nope=128, qk_rope=64, v_head=128, dense_inter=3 * hidden, first_k_dense=1, n_routed=experts, top_k=TOP,
                    n_shared=1, moe_inter=ff, scoring="sigmoid", norm_topk_prob=False)
    return g, k


def fasodra_pair(hidden: int):
    """(Fasodra, neighbour) of one size: 128-wide attention heads, 64-wide time-mixing heads over the whole width, half as many delta heads as the
    neighbour, ungated experts of the neighbour's parameter count.  Chunks of 5120: the 8k context ends 3072 tokens into one."""
    heads, kv, experts, ff, vocab = hidden // 128, max(1, hidden // 512), hidden // 64, hidden * 3 // 4, 65536
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": TOP}}
    base = {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5}
    lft = base | {"rot": {"base": 1e5, "dims": 64}}
    kinds = [("attention", base | {"bias_max": 4096, "mask": {"size": 5120}}),
             ("parallel", {"left": lft, "right": {"heads": hidden // 64, "dim": 64}, "left_scale": 0.7, "right_scale": 0.9}),
             ("attention", base | {"bias_max": 4096, "mask": {"size": 5120}}),
             ("parallel_2", {"left": lft, "right": {"heads": heads, "kv_heads": heads, "dim": 128, "vdim": 128, "conv": 4}})]
    f = fasodra_config({"name": f"fasodra-{hidden}", "vocab": vocab, "width": hidden, "norm": {"eps": 1e-5}, "residual_mult": 0.8, "streams": 2,
                        "layers": [{"type": kinds[i % 4][0], "mixer": kinds[i % 4][1], "mlp": mlp} for i in range(N_LAYERS)]})
    return f, gazutar_pair(hidden)[0]


def nivasun_set(hidden: int):
    """(Nivasun, neighbours) of one size: 128-wide heads, attention, latent attention and differential attention (half the heads, two maps and 256 value
    channels each) in turns over windows of half the context; six layers, the second and third run twice, so that there are as many layer runs as layers in
    the neighbours."""
    heads, kv, experts, ff, vocab = hidden // 128, max(1, hidden // 512), hidden // 64, hidden // 2, 65536
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": TOP}, "shared": {"ff": ff}}
    rot, base = {"base": 1e5, "dims": 128}, {"dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 4096}}
    kinds = [("attention", base | {"heads": heads, "kv_heads": kv, "rot": rot}), ("latent_attention", base | {"heads": heads, "kv_rank": 512, "q_rank": hidden * 3 // 8}),
             ("attention_2", base | {"heads": heads // 2, "kv_heads": max(1, kv // 2), "vdim": 256, "diff": 0.5, "rot": rot})]
    n = nivasun_config({"name": f"nivasun-{hidden}", "vocab": vocab, "width": hidden, "norm": {"eps": 1e-5}, "canon": {"taps": 4}, "logit_softcap": 30.0,
                        "embedding": {"scale": 1.0, "bigram": {"buckets": vocab, "mul_prev": 53, "mul_cur": 29}}, "loop": {"start": 1, "stop": 3, "times": 2},
                        "layers": [{"type": kinds[i % 3][0], "mixer": kinds[i % 3][1], "mlp": mlp} for i in range(N_LAYERS - 2)]})
    return n, rubasun_pair(hidden)[0], gazutar_pair(hidden)[0]


DESIGNS = {"gazutar": gazutar_pair, "rubasun": rubasun_pair, "fasodra": fasodra_pair, "nivasun": nivasun_set}


def _peaks():
    p = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    if os.path.exists(p):
        d = json.load(open(p))
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12
    return 6.65e12, 1.59e15


def _events(fn, stream, reps):
    out = []
    with torch.cuda.stream(stream):
        for _ in range(3):
            fn()
        for _ in range(reps):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record(stream)
            fn()
            b.record(stream)
            stream.synchronize()
            out.append(a.elapsed_time(b))
    return statistics.median(out)


def launcher_times(eng, run, reps=5) -> dict:
    """{launcher: (calls per step, microseconds per call)} of the step that ``run`` launches eagerly."""
    calls, orig = [], nat.call

    def rec(name, *a, **k):
        if nat.SIGS[name][1]:
            calls.append((name, a))
        return orig(name, *a, **k)

    with torch.cuda.stream(eng.stream):
        run()
        nat.call = rec
        try:
            run()
        finally:
            nat.call = orig
        eng.stream.synchronize()
        out = {}
        for name in dict.fromkeys(n for n, _ in calls):
            mine = [a for n, a in calls if n == name]
            g = torch.cuda.CUDAGraph()
            loops = 1 if len(mine) > 4 else 4
            with torch.cuda.graph(g, stream=eng.stream):
                for _ in range(loops):
                    for a in mine:
                        orig(name, *a)
            out[name] = (len(mine), round(_events(g.replay, eng.stream, reps) * 1e3 / (len(mine) * loops), 2))
            del g
    return out


def work(cfg, rows: int, ctx: int, batch: int) -> dict:
    """{launcher: ("bytes" | "flops", amount per call)} of the operations that have a clear floor."""
    H = cfg.hidden
    heads = cfg.kda_heads
    out = {}
    state = 2 * batch * heads * 128 * 128 * 4                       # read and write the recurrent state once
    gates = 2 * heads * 128 * 128 * 2
    per_tok = heads * (4 * 128 * 128 + 6 * 64 * 128) * 2            # chunk form: state products, pair products
    decode = rows == batch
    rec = ("bytes", state + gates + rows * heads * 128 * 18) if decode else ("flops", rows * per_tok)
    mixers = [x for i, _ in cfg.layer_runs() for x in cfg.blocks[i].mixers] if cfg.blocks else []
    att = next((x for x in mixers if not x.recurrent), None)
    lat, rot, ah, dn, dv = cfg.kv_lora, cfg.qk_rope, cfg.n_heads, cfg.qk_nope, cfg.v_head
    lw = min([b.window or ctx for b in mixers if b.latent], default=ctx)
    seen = sum(min(p + 1, lw) for p in range(ctx - rows, ctx)) / rows      # keys a row of the chunk sees on average
    latent = ("bytes", batch * min(ctx, lw) * (lat + rot) * 2 + rows * ah * (2 * lat + rot) * 2) if decode else ("flops", 2 * rows * seen * ah * (2 * lat + rot))
    # the queries' way into the latent space and the values' way out of it: weights and activations, or products
    absorb, up = ((("bytes", ah * lat * d * 2 + rows * ah * (lat + d) * 2) if decode else ("flops", 2 * rows * ah * lat * d)) for d in (dn, dv))
    experts = TOP + cfg.n_shared
    if any(b.latent for b in mixers):
        out["lsb_latent_attn"], out["lsb_latent_query"], out["lsb_latent_out"] = latent, absorb, up
        out["lsb_latent_expand"] = ("flops", 2 * min(ctx, lw + rows) * ah * lat * (dn + dv))
        out["lsb_attn_run"] = ("flops", 2 * rows * seen * ah * (dn + rot + dv))
        out["lsb_resid_update"] = ("bytes", rows * H * 14)
        out["lsb_glu"] = ("bytes", rows * cfg.moe_inter * 10)
    if any(b.softmax for b in mixers):
        mean = lambda xs: sum(xs) / max(1, len(xs))
        keys = lambda b: min(ctx % b.chunk or b.chunk if b.chunk else ctx, b.window or ctx)            # that a decoded token sees
        per_row = lambda b: mean([min(p % b.chunk + 1 if b.chunk else p + 1, b.window or ctx) for p in range(ctx - rows, ctx)])
        soft = [b for b in mixers if b.softmax]
        kv = lambda b: b.kv_heads * (b.maps * b.dim + b.vdim) * 2
        out["lsb_attn"] = (("bytes", mean([batch * keys(b) * kv(b) + rows * b.heads * b.vdim * (6 if b.out_gate else 4) for b in soft])) if decode
                           else ("flops", mean([2 * rows * per_row(b) * b.heads * b.maps * (b.dim + b.vdim) for b in soft])))
        out["lsb_attn_prep"] = out["lsb_attn_head_prep"] = ("bytes", mean([rows * ((b.heads + b.kv_heads) * b.maps * b.dim * 6 + b.kv_heads * b.vdim * (2 if b.shared_kv else 6))
                                                                          for b in soft]))
        out["lsb_attn_diff"] = ("bytes", mean([rows * b.heads * b.vdim * 10 for b in soft if b.maps > 1]))
        out["lsb_resid_update"] = ("bytes", rows * H * (14 + TOP * 4) // 2 + rows * H * 7)
        # chunk form: two state products and two (delta rule: six, with the solve) products over pairs of a chunk
        dlt, tm = [b for b in mixers if b.delta], [b for b in mixers if b.kind == "time_mix"]
        st = lambda b: 2 * batch * b.heads * b.dim * b.vdim * 4                                        # the state read and written once
        if decode:
            low = lambda b: b.heads * (b.dim + b.vdim) * 128 * 2 if b.kind == "channel_delta" else 0
            out["lsb_delta_forward"] = ("bytes", mean([st(b) + low(b) + rows * b.heads * b.dim * 18 for b in dlt]))
            out["lsb_tmix_forward"] = ("bytes", mean([st(b) + b.heads * b.dim * b.dim * 2 + rows * b.heads * b.dim * 18 for b in tm]))
        else:
            out["lsb_delta_forward"] = ("flops", mean([rows * b.heads * (4 * b.dim * b.vdim + 6 * 64 * b.dim) * 2 for b in dlt]))
            out["lsb_tmix_forward"] = ("flops", mean([rows * b.heads * (2 * b.dim * b.vdim + 2 * 64 * b.dim) * 2 for b in tm]))
        out["lsb_tmix_shift"] = ("bytes", rows * H * 12)
        n = cfg.streams
        ups = [rows * H * (4 + 4 * n + 2)] + [rows * H * (8 * n + 2 + s) for b in cfg.blocks for s in ((8 if b.join == "normed" and b.branches else 4), TOP * 4)]
        out["lsb_stream_update"] = ("bytes", mean(ups))
    if cfg.norm_place == "parallel":
        # one update per layer run and one in front of the first; steps of single tokens have the convolution in it (its state read and written)
        out["lsb_resid_update"] = ("bytes", rows * H * (14 + TOP * 4 + ((2 + 8 * (cfg.input_conv - 1)) if decode else 0)))
        out["lsb_input_conv"] = ("bytes", rows * H * 4)
        out["lsb_glu"] = ("bytes", rows * cfg.moe_inter * 10)
    if att is None:
        out["lsb_kda_forward"] = out["lsb_kda_forward_chunked"] = rec
        out["lsb_mla_decode"] = latent
        out["lsb_batched_gemv_bf16"] = (absorb[0], (absorb[1] + up[1]) / 2)
        out["lsb_add_rmsnorm"] = ("bytes", rows * H * 14)
        out["lsb_moe_combine"] = ("bytes", rows * H * (experts + 1) * 4)
        out["lsb_mla_prep"] = ("bytes", rows * (cfg.q_lora + lat + rot) * 6)
    if rows == 1:                          # (how many experts a batch touches is the router's affair)
        by = experts * 3 * H * cfg.moe_inter * 2
        out["lsb_moe_up"] = ("bytes", by / 3)
        out["lsb_moe_gateup"] = out["lsb_moe_gateup_act"] = ("bytes", by * 2 / 3)
        out["lsb_moe_down"] = ("bytes", by / 3)
    elif rows > 1024:
        own = cfg.blocks and (cfg.blocks[-1].scale_input or cfg.blocks[-1].unit != "glu")      # up and down are one size, or gate/up is a launcher of its own
        out["lsb_moe_tc_ffn"] = ("flops", (2 if own else 3) * rows * experts * H * cfg.moe_inter)
        out["lsb_moe_tc_gateup_act"] = ("flops", 4 * rows * experts * H * cfg.moe_inter)
    return out


def measure(cfg, ctx: int, chunk: int, batches, clocks=None) -> dict:
    hbm, tf = _peaks()
    dev = torch.device("cuda", torch.cuda.current_device())
    m = model_class(cfg).random_init(cfg, dev, "bf16", 64, seed=5)
    bmax = max(batches)
    eng = Engine(m, max_seqs=bmax, max_ctx=ctx + chunk + 256, prefill_chunk=chunk, max_batch=bmax)
    g = torch.Generator().manual_seed(1)
    tok = lambda n: torch.randint(0, cfg.vocab, (n,), generator=g).tolist()
    res: dict = {"model": cfg.name, "weight_gib": round(m.weight_bytes() / 2 ** 30, 2)}

    def table(times, rows, batch):
        w = work(cfg, rows, ctx, batch)
        t = {}
        for k, (n, us) in sorted(times.items(), key=lambda x: -x[1][0] * x[1][1]):
            e = {"calls": n, "us": us}
            if k in w:
                kind, amount = w[k]
                e["of_measured_" + ("hbm" if kind == "bytes" else "bf16")] = round(amount / (us * 1e-6) / (hbm if kind == "bytes" else tf), 4)
            t[k] = e
        return t

    warm = eng.create_sequence()
    eng.prefill(warm, tok(chunk))
    eng.free_sequence(warm)
    s0 = eng.create_sequence()
    eng.prefill(s0, tok(ctx - chunk))
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record(eng.stream)
    nxt = eng.prefill(s0, tok(chunk))
    e1.record(eng.stream)
    torch.cuda.synchronize()
    ms = e0.elapsed_time(e1)
    res["prefill"] = {"chunk": chunk, "context": ctx, "ms": round(ms, 3), "tok_s": round(chunk / ms * 1e3, 1)}
    ws = eng.ws_prefill                       # still staged with the last chunk
    res["prefill"]["launchers"] = table(launcher_times(eng, lambda: m.forward(ws, chunk, 1, chunk - 1, 1)), chunk, 1)
    sids, toks = [s0], [nxt]
    res["decode"] = {}
    for B in batches:
        while len(sids) < B:
            sids.append(eng.create_sequence())
            toks.append(eng.prefill(sids[-1], tok(ctx)))
        for _ in range(4):
            toks = eng.decode(sids, toks)
        n = 32
        e0.record(eng.stream)
        for _ in range(n):
            toks = eng.decode(sids, toks)
        e1.record(eng.stream)
        torch.cuda.synchronize()
        e2e = e0.elapsed_time(e1) / n
        wd = eng.ws_decode[B]
        dev_ms = _events(eng.graphs[B].replay, eng.stream, 20)
        res["decode"][str(B)] = {"ms_per_step": round(dev_ms, 4), "tok_s": round(B / dev_ms * 1e3, 1), "e2e_tok_s": round(B / e2e * 1e3, 1),
                                 "launchers": table(launcher_times(eng, lambda: m.forward(wd, B, B, 0, B)), B, B)}
    del eng, m
    torch.cuda.empty_cache()
    return res


def run(design: str, sizes, ctx: int = 8192, chunk: int = 2048, batches=(1, 32), sampler=None) -> dict:
    pair = DESIGNS[design]
    out = {"metric": "prefill and decode throughput beside the closest design", "design": design, "data": "random weights, synthetic token ids", "dtype": "bf16",
           "context": ctx, "l2": "decode and prefill steps stream more weights than L2 holds", "sizes": {}}
    if sampler is not None:
        sampler.start()
    for h in sizes:
        out["sizes"][str(h)] = [measure(c, ctx, chunk, list(batches)) for c in pair(h)]
    if sampler is not None:
        out["clocks"] = sampler.stop()
    return out
