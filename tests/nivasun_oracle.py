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
