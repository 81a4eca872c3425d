"""Plain evaluation of the Nivasun design, one function per mechanism, used as the oracle of the device path.

Whole sequences at a time, in the type of the tensors, from a ``config.json`` dictionary and a dictionary of tensors under the checkpoint's own
names.  No code is shared with the package.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------------------------------------ embedding, norms, convolution
def rms(x, eps):
    return x / torch.sqrt(x.square().mean(-1, keepdim=True) + eps)


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the bigram table for every token of a sequence; the first token has the last row."""
    t = [int(x) for x in tokens]
    return [buckets] + [(a * mul_prev + b * mul_cur) % buckets for a, b in zip(t, t[1:])]


def embed(cfg, w, tokens):
    e, b = cfg["embedding"], cfg["embedding"]["bigram"]
    rows = bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])
    return w["embed"][torch.as_tensor(tokens)] * e["scale"] + w["bigram"][torch.tensor(rows)]


def input_conv(h, taps):
    """h [T, C], taps [C, n], last column = current token; zeros before the start."""
    n = taps.shape[1]
    y = torch.cat([torch.zeros(n - 1, h.shape[1], dtype=h.dtype), h])
    return sum(y[j: j + len(h)] * taps[:, j] for j in range(n))


# ------------------------------------------------------------------------------------------------ attention
def visible(T, window):
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < window)


def _turn(x, base, dims, first, second):
    """Channels ``first`` and ``second`` of x [T, heads, d] turned as pairs by position * base^(-2 i / dims)."""
    f = torch.tensor([base ** (-2 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None, None] * f
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v, y = x[..., first], x[..., second], x.clone()
    y[..., first], y[..., second] = u * c - v * s, v * c + u * s
    return y


def rotate_half(x, dims, base):
    return _turn(x, base, dims, slice(0, dims // 2), slice(dims // 2, dims))


def rotate_pairs(x, dims, base):
    return _turn(x, base, dims, slice(0, dims, 2), slice(1, dims, 2))


def softmax_with_sink(s, sink):
    """s [H, T, T] with -inf where nothing is seen; ``sink`` [H]: one more term of the denominator."""
    m = torch.maximum(s.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - m))


def attend(q, k, v, scale, window, temp=None, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; temp, sink [H]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, 1)) * scale
    if temp is not None:
        s = s * temp[:, None, None]
    s = s.masked_fill(~visible(T, window), float("-inf"))
    p = torch.softmax(s, -1) if sink is None else softmax_with_sink(s, sink)
    return torch.einsum("hij,jhe->ihe", p, v.repeat_interleave(H // G, 1))


def attention_mixer(m, eps, w, p, h):
    """The values are the keys as projected."""
    T, H, G, d = len(h), m["heads"], m["kv_heads"], m["dim"]
    q, k = (h @ w[p + "q"].T).view(T, H, d), (h @ w[p + "k"].T).view(T, G, d)
    r = lambda x: rotate_half(x, m["rot"]["dims"], m["rot"]["base"])
    return attend(r(q), r(k), k, m["scale"], m["mask"]["size"], w[p + "temp"], w[p + "sink"]).flatten(1) @ w[p + "o"].T


def latent_mixer(m, eps, w, p, h):
    T, H = len(h), m["heads"]
    q = (rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T
    c = rms(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]
    k, v = (c @ w[p + "uk"].T).view(T, H, m["dim"]), (c @ w[p + "uv"].T).view(T, H, m["vdim"])
    o = attend(q.view(T, H, m["dim"]), k, v, m["scale"], m["mask"]["size"])
    return (o.flatten(1) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def map_weight(m, w, p):
    """The factor of the second map of a differential attention."""
    s = [(w[p + "lq" + n] * w[p + "lk" + n]).sum() for n in "12"]
    return torch.exp(s[0]) - torch.exp(s[1]) + m["diff"]


def differential_mixer(m, eps, w, p, h):
    T, H, G, d, e = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    r = lambda x: rotate_pairs(x, m["rot"]["dims"], m["rot"]["base"])
    q, k = (h @ w[p + "q"].T).view(T, H, 2, d), (h @ w[p + "k"].T).view(T, G, 2, d)
    v = (h @ w[p + "v"].T).view(T, G, e)
    a = [attend(r(q[:, :, i]), r(k[:, :, i]), v, m["scale"], m["mask"]["size"]) for i in (0, 1)]
    o = rms(a[0] - map_weight(m, w, p) * a[1], eps) * (1.0 - m["diff"])
    return o.flatten(1) @ w[p + "o"].T


MIXERS = {"attention": attention_mixer, "latent_attention": latent_mixer, "attention_2": differential_mixer}


# ------------------------------------------------------------------------------------------------ experts
def silu(x):
    return x * torch.sigmoid(x)


def expert(w, p, x):
    return (silu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def route(logits, top):
    """(ids, weights) [T, top]: the largest logits, softmax over those alone."""
    z, ids = logits.topk(top, dim=-1)
    return ids, torch.softmax(z, -1)


def moe(m, w, p, h):
    ids, wt = route(h @ w[p + "router"].T + w[p + "router.b"], m["router"]["top"])
    y = torch.sigmoid(h @ w[p + "shared.sg"].T) * expert(w, p + "shared.", h)
    for e in range(m["router"]["experts"]):
        t, s = torch.nonzero(ids == e, as_tuple=True)
        if len(t):
            y[t] += wt[t, s][:, None] * expert(w, p + f"e{e}.", h[t])
    return y


# ------------------------------------------------------------------------------------------------ whole model
def layer(cfg, w, i, x):
    L, p, eps = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"]
    h = rms(x, eps) * w[p + "norm1"]
    y = MIXERS[L["type"]](L["mixer"], eps, w, p + "mix.", h + input_conv(h, w[p + "canon1"]))
    return x + y + (moe(L["mlp"], w, p + "mlp.", h) if L.get("mlp") else 0.0)


def layer_runs(cfg):
    """[(layer, number of the pass that starts in front of it or None)] in the order in which the layers run."""
    n, lp = len(cfg["layers"]), cfg["loop"]
    inner = [(i, t if i == lp["start"] else None) for t in range(lp["times"]) for i in range(lp["start"], lp["stop"])]
    return [(i, None) for i in range(lp["start"])] + inner + [(i, None) for i in range(lp["stop"], n)]


def forward(cfg, w, tokens, want_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer run)."""
    x, layers = embed(cfg, w, tokens), []
    for i, t in layer_runs(cfg):
        if t is not None:
            x = x + w["loop.step"][t]
        x = layer(cfg, w, i, x)
        layers.append(x)
    lg = (rms(x, cfg["norm"]["eps"]) * w["final.norm"]) @ w["head"].T
    c = cfg["logit_softcap"]
    lg = c * torch.tanh(lg / c)
    return (lg, layers) if want_layers else lg


# ------------------------------------------------------------------------------------------------ random models
def random_model(cfg, seed=0, close_calls=True):
    """Tensors for a configuration, spread so that every mechanism matters.  Without ``close_calls`` the router's bias decides the choice (rounding cannot
    turn it)."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    u = lambda lo, hi, *s: lo + (hi - lo) * torch.rand(s, generator=g)
    H, V, w = cfg["width"], cfg["vocab"], {}
    lin = lambda o, i: n(o, i) / i ** 0.5
    w["embed"], w["head"] = n(V, H) / cfg["embedding"]["scale"], 2.0 * lin(V, H)
    w["bigram"], w["loop.step"], w["final.norm"] = 0.7 * n(cfg["embedding"]["bigram"]["buckets"] + 1, H), 0.7 * n(cfg["loop"]["times"], H), u(0.8, 1.3)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        x, h, d, e = p + "mix.", m["heads"], m["dim"], m["vdim"]
        w[p + "norm1"], w[p + "canon1"] = u(0.7, 1.4), u(-0.7, 0.7, H, cfg["canon"]["taps"])
        if L["type"] == "attention":
            w[x + "q"], w[x + "k"] = 1.5 * lin(h * d, H), 1.5 * lin(m["kv_heads"] * d, H)
            w[x + "temp"], w[x + "sink"] = u(0.4, 1.8, h), 1.5 * n(h)
        elif L["type"] == "latent_attention":
            w[x + "dq"], w[x + "dkv"], w[x + "dq.norm"], w[x + "dkv.norm"] = lin(m["q_rank"], H), lin(m["kv_rank"], H), 1.0 + 0.2 * n(m["q_rank"]), 1.0 + 0.2 * n(m["kv_rank"])
            w[x + "uq"], w[x + "uk"], w[x + "uv"], w[x + "g"] = 1.5 * lin(h * d, m["q_rank"]), 1.5 * lin(h * d, m["kv_rank"]), lin(h * e, m["kv_rank"]), lin(h * e, H)
        else:
            w[x + "q"], w[x + "k"], w[x + "v"] = 1.5 * lin(h * 2 * d, H), 1.5 * lin(m["kv_heads"] * 2 * d, H), lin(m["kv_heads"] * e, H)
            w |= {x + t: 0.6 * n(d) / d ** 0.5 for t in ("lq1", "lk1", "lq2", "lk2")}
        w[x + "o"] = lin(H, h * e)
        if L.get("mlp"):
            z, E, f, sf = p + "mlp.", L["mlp"]["router"]["experts"], L["mlp"]["expert"]["ff"], L["mlp"]["shared"]["ff"]
            w[z + "router"], w[z + "router.b"] = lin(E, H), 0.7 * n(E)
            if not close_calls:
                w[z + "router"], w[z + "router.b"] = 0.1 * w[z + "router"], torch.randperm(E, generator=g).float()
            for q, c in [(f"e{j}.", f) for j in range(E)] + [("shared.", sf)]:
                w[z + q + "gate"], w[z + q + "up"], w[z + q + "down"] = 1.5 * lin(c, H), lin(c, H), lin(H, c)
            w[z + "shared.sg"] = lin(1, H)
    return w


def att(heads, kv_heads, dim, window, rot, base=10000.0, mlp=None, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale or round(1.3 / dim ** 0.5, 4), "mask": {"size": window},
                                           "rot": {"base": base, "dims": rot}}, "mlp": mlp}


def lat(heads, dim, vdim, kv_rank, q_rank, window, mlp=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": round(1.3 / dim ** 0.5, 4),
                                                  "mask": {"size": window}}, "mlp": mlp}


def dif(heads, kv_heads, dim, vdim, window, rot, diff, base=10000.0, mlp=None):
    return {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": round(1.3 / dim ** 0.5, 4), "diff": diff,
                                             "mask": {"size": window}, "rot": {"base": base, "dims": rot}}, "mlp": mlp}


def moe_spec(experts, top, ff, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}


def model_cfg(width, vocab, layers, loop, taps, bigram, eps=1e-5, cap=12.0, scale=3.0):
    return {"architecture": "Nivasun", "canon": {"taps": taps}, "embedding": {"scale": scale, "bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "layers": layers,
            "logit_softcap": cap, "loop": dict(zip(("start", "stop", "times"), loop)), "norm": {"eps": eps}, "vocab": vocab, "width": width}


# several geometries: every kind first, last, inside and outside the loop, layers without a feed-forward, loops at either end and of a single pass,
# sizes off the kernels' tiles and on them, sizes of one, heads wider than the tensor-core forms take, one tap and many
MODELS = {
    "odd": lambda: model_cfg(136, 301, [lat(5, 20, 12, 44, 36, 33, moe_spec(5, 2, 40, 24)), att(6, 2, 24, 21, 10, 500.0, moe_spec(7, 3, 24, 40)),
                                        dif(6, 3, 20, 36, 26, 12, 0.35, 300.0), att(3, 3, 40, 70, 40), dif(4, 1, 12, 20, 17, 12, 0.7, 77.0, moe_spec(4, 1, 56, 9))],
                             (1, 3, 2), 4, (97, 1000003, 12345), 3e-3, 9.0),
    "tiles": lambda: model_cfg(384, 520, [dif(4, 4, 64, 128, 130, 64, 0.5, 1e6, moe_spec(12, 4, 128, 256)), att(16, 2, 128, 64, 64, 1e6, moe_spec(12, 4, 128, 128)),
                                          lat(8, 64, 96, 128, 112, 90, moe_spec(12, 4, 256, 128)), att(8, 8, 64, 48, 32, mlp=moe_spec(8, 3, 128, 128))], (0, 2, 2), 3, (1024, 31, 7)),
    "ones": lambda: model_cfg(48, 40, [att(1, 1, 2, 1, 2, mlp=moe_spec(1, 1, 1, 1)), lat(1, 1, 1, 1, 1, 9, moe_spec(3, 3, 8, 5)), dif(1, 1, 2, 3, 2, 2, 0.2),
                                       dif(2, 2, 8, 8, 33, 4, 0.9, 5.0)], (0, 4, 1), 1, (1, 1, 1), 1e-6, 30.0, 1.0),
    "wide": lambda: model_cfg(250, 200, [att(33, 1, 24, 90, 24, 60.0, moe_spec(4, 1, 96, 30)), lat(3, 136, 200, 540, 100, 60, moe_spec(6, 2, 64, 64)), dif(2, 1, 264, 72, 41, 100, 0.45),
                                         att(2, 2, 272, 55, 128), lat(20, 40, 24, 200, 250, 128), dif(5, 5, 16, 280, 64, 10, 0.6, 1e5, moe_spec(6, 5, 32, 100))],
                              (4, 6, 3), 6, (509, 53, 29), 1e-4),
}
