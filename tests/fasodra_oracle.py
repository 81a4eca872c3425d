"""Plain evaluation of the Fasodra design, one function per mechanism, used as the oracle of the device path.

Whole sequences at a time, recurrences token by token, from a ``config.json`` dictionary and a dictionary of tensors under the checkpoint's own
names, in the type of the tensors.  No code is shared with the package.
"""
from __future__ import annotations

import math

import torch

UNIT_EPS = 1e-6            # inside the square root of the delta rule's unit vectors


# ------------------------------------------------------------------------------------------------ norms, streams
def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt(d.square().mean(-1, keepdim=True) + eps) * w + b


def rms(x, eps):
    return x / torch.sqrt(x.square().mean(-1, keepdim=True) + eps)


def read_streams(streams, w_in):
    """streams: list of [T, width]; the sublayer's input in front of its norm."""
    return sum(w_in[s] * x for s, x in enumerate(streams))


def write_streams(streams, mix, out, y):
    """New streams from the old ones (mix indexed [from, to]) and a sublayer's scaled output."""
    n = len(streams)
    return [sum(mix[s, t] * streams[s] for s in range(n)) + out[t] * y for t in range(n)]


# ------------------------------------------------------------------------------------------------ attention
def bucket(n, rows, reach):
    """Bucket of a distance: one each up to half the rows, then logarithmic up to ``reach``, then the last."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half) + 1e-9))


def distance_bias(table, T, reach):
    """[H, T, T]: entry (h, i, j) is the bias of distance i - j (entries with j > i are not used)."""
    of = torch.tensor([bucket(n, table.shape[0], reach) for n in range(T)])
    dist = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)
    return table[of[dist]].permute(2, 0, 1)


def visible(T, chunk=0):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i // chunk == j // chunk) if chunk else torch.ones_like(i - j, dtype=torch.bool))


def attention(q, k, v, scale, bias=None, chunk=0):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, 1)) * scale
    if bias is not None:
        s = s + bias
    p = torch.softmax(s.masked_fill(~visible(T, chunk), float("-inf")), -1)
    return torch.einsum("hij,jhe->ihe", p, v.repeat_interleave(H // G, 1))


def rotate_half(x, dims, base):
    """Rotary embedding of the first ``dims`` channels of x [T, heads, d]: channel i turns with channel i + dims / 2."""
    n = dims // 2
    f = torch.tensor([base ** (-2 * i / dims) for i in range(n)], dtype=torch.float64)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None, None] * f
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., :n], x[..., n: dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def attention_heads(spec, eps, w, p, h, norm=None, rotary=False, chunk=0, rel=None):
    """Heads [T, H, e] of an attention mixer in front of its output projection.  norm: None, "plain" (no weight) or "weight"."""
    T, H, G, d, e = len(h), spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q, k, v = ((h @ w[p + n].T + w[p + n + ".b"]).view(T, m, c) for n, m, c in (("q", H, d), ("k", G, d), ("v", G, e)))
    if norm:
        q, k = rms(q, eps), rms(k, eps)
    if norm == "weight":
        q, k = q * w[p + "q.norm"], k * w[p + "k.norm"]
    if rotary:
        q, k = (rotate_half(t, spec["rot"]["dims"], spec["rot"]["base"]) for t in (q, k))
    return attention(q, k, v, spec["scale"], None if rel is None else distance_bias(rel, T, spec["bias_max"]), chunk)


def chunked_mixer(spec, eps, w, p, h):
    o = attention_heads(spec, eps, w, p, h, "plain", chunk=spec["mask"]["size"], rel=w[p + "rel"])
    return o.flatten(1) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ recurrences
def token_shift(h, mu):
    return h + (torch.cat([torch.zeros_like(h[:1]), h[:-1]]) - h) * mu


def time_mixing(r, k, v, w, u, S=None):
    """r, k, w [T, H, d], v [T, H, e], u [H, d] -> ([T, H, e], state [H, d, e]); the bonus u counts for the current token only."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[2], dtype=r.dtype) if S is None else S
    out = torch.empty_like(v)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hde,hd->he", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    return out, S


def silu(x):
    return x * torch.sigmoid(x)


def time_mixer(spec, eps, w, p, h):
    T, H, d = len(h), spec["heads"], spec["dim"]
    x = {n: token_shift(h, w[p + "mu." + n]) for n in "rkvgw"}
    r, k, v = ((x[n] @ w[p + n].T).view(T, H, d) for n in "rkv")
    decay = torch.exp(-torch.exp(torch.tanh(x["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).view(T, H, d)
    o, _ = time_mixing(r, k, v, decay, w[p + "u"])
    return (rms(o, eps).flatten(1) * w[p + "norm"] * silu(x["g"] @ w[p + "g"].T)) @ w[p + "o"].T


def short_conv(x, taps):
    """x [T, C], taps [C, n], last column = current token; zeros before the start; then silu."""
    n = taps.shape[1]
    y = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x])
    return silu(sum(y[j: j + len(x)] * taps[:, j] for j in range(n)))


def unit(x):
    return x / torch.sqrt(x.square().sum(-1, keepdim=True) + UNIT_EPS)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def delta_rule(q, k, v, g, beta, S=None):
    """q, k [T, H, d], v [T, H, e], g, beta [T, H] -> ([T, H, e], state [H, d, e]); decay, read, write, read out."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if S is None else S
    out = torch.empty_like(v)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hde,hd->he", S, q[t])
    return out, S


def delta_mixer(spec, eps, w, p, h):
    T, H, G, d, e = len(h), spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q, k, v = (short_conv(h @ w[p + n].T, w[p + n + ".conv"]) for n in "qkv")
    q, k = (unit(t.view(T, G, d)).repeat_interleave(H // G, 1) for t in (q, k))
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o, _ = delta_rule(q * d ** -0.5, k, v.view(T, H, e), g, torch.sigmoid(h @ w[p + "b"].T))
    return ((rms(o, eps) * w[p + "norm"]).flatten(1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ side by side
def parallel_mixer(spec, eps, w, p, h):
    """Gated rotary attention beside time mixing, a constant factor on each."""
    s = spec["left"]
    o = attention_heads(s, eps, w, p + "left.", h, rotary=True) * torch.sigmoid(h @ w[p + "left.g"].T)[..., None]
    return spec["left_scale"] * (o.flatten(1) @ w[p + "left.o"].T) + spec["right_scale"] * time_mixer(spec["right"], eps, w, p + "right.", h)


def parallel_2_mixer(spec, eps, w, p, h):
    """Normed rotary attention beside a delta rule, each result normed, the mean of both."""
    a = attention_heads(spec["left"], eps, w, p + "left.", h, "weight", rotary=True).flatten(1) @ w[p + "left.o"].T
    b = delta_mixer(spec["right"], eps, w, p + "right.", h)
    return 0.5 * (rms(a, eps) * w[p + "left.out"] + rms(b, eps) * w[p + "right.out"])


MIXERS = {"attention": chunked_mixer, "parallel": parallel_mixer, "parallel_2": parallel_2_mixer}


# ------------------------------------------------------------------------------------------------ experts
def route(logits, top):
    """(ids, weights) [T, top]: softmax scores of the best, divided by their sum."""
    s, ids = torch.softmax(logits, -1).topk(top, dim=-1)
    return ids, s / (s.sum(-1, keepdim=True) + 1e-20)


def expert(w, p, x):
    return torch.relu(x @ w[p + "up"].T).square() @ w[p + "down"].T


def moe(spec, w, p, h):
    ids, wt = route(h @ w[p + "router"].T, spec["router"]["top"])
    y = torch.zeros_like(h)
    for t in range(len(h)):
        for i, c in zip(ids[t].tolist(), wt[t]):
            y[t] += c * expert(w, p + f"e{i}.", h[t: t + 1])[0]
    return y


def forward(cfg, w, tokens, want_layers=False):
    """Logits [T, vocab] of one sequence (and the sum of the streams after every layer)."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens)]
    xs, layers = [x] * cfg["streams"], []

    def sublayer(xs, p, q, f):
        h = layer_norm(read_streams(xs, w[f"{p}hc{q}.in"]), w[f"{p}norm{q}"], w[f"{p}norm{q}.b"], eps)
        return write_streams(xs, w[f"{p}hc{q}.mix"], w[f"{p}hc{q}.out"], m * f(h))

    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        xs = sublayer(xs, p, 1, lambda h: MIXERS[L["type"]](L["mixer"], eps, w, p + "mix.", h))
        if L.get("mlp"):
            xs = sublayer(xs, p, 2, lambda h: moe(L["mlp"], w, p + "mlp.", h))
        layers.append(sum(xs))
    lg = layer_norm(sum(xs), w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
    return (lg, layers) if want_layers else lg


# ------------------------------------------------------------------------------------------------ random models
def random_model(cfg, seed=0, close_calls=True, rel_rows=(32, 10, 6), rank=12):
    """Tensors for a configuration, spread so that every mechanism matters.  ``rel_rows``: rows of the distance bias tables, in turns.  Without
    ``close_calls`` the bias of the norm in front of a router decides the choice (rounding cannot turn it)."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    u = lambda lo, hi, *s: lo + (hi - lo) * torch.rand(s, generator=g)
    H, V, S, w = cfg["width"], cfg["vocab"], cfg["streams"], {}
    lin = lambda o, i: n(o, i) / i ** 0.5

    def norm(p):
        w[p], w[p + ".b"] = 1.0 + 0.2 * n(H), 0.3 * n(H)

    def attn(p, m, gate=False, weight=False):
        for t, c in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
            w[p + t], w[p + t + ".b"] = 1.5 * lin(c, H), 0.4 * n(c)
        if weight:
            w[p + "q.norm"], w[p + "k.norm"] = 1.5 * (1.0 + 0.2 * n(m["dim"])), 1.0 + 0.2 * n(m["dim"])
        if gate:
            w[p + "g"] = lin(m["heads"], H)
        w[p + "o"] = lin(H, m["heads"] * m["vdim"])

    def time(p, m):
        c = m["heads"] * m["dim"]
        for t in "rkvgw":
            w[p + "mu." + t] = u(0.1, 0.9, H)
        for t in "rkvg":
            w[p + t] = lin(c, H)
        w[p + "w1"], w[p + "w2"], w[p + "w0"], w[p + "u"] = lin(rank, H), 1.5 * lin(c, rank), u(-5.0, 0.5, c), 0.7 * n(m["heads"], m["dim"])
        w[p + "norm"], w[p + "o"] = 1.0 + 0.2 * n(c), lin(H, c)

    def delta(p, m):
        h, k, v = m["heads"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
        for t, c in (("q", k), ("k", k), ("v", v)):
            w[p + t], w[p + t + ".conv"] = lin(c, H), u(-1.0, 1.0, c, m["conv"])
        w[p + "b"], w[p + "a"], w[p + "g"], w[p + "o"] = lin(h, H), lin(h, H), lin(v, H), lin(H, v)
        w[p + "A_log"], w[p + "dt_bias"], w[p + "norm"] = u(-3.0, 0.5, h), u(-3.0, 0.0, h), 1.0 + 0.2 * n(m["vdim"])

    w["embed"], w["head"] = n(V, H), lin(V, H)
    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        x = p + "mix."
        norm(p + "norm1")
        if L["type"] == "attention":
            attn(x, m)
            w[x + "rel"] = n(rel_rows[i % len(rel_rows)], m["heads"])
        elif L["type"] == "parallel":
            attn(x + "left.", m["left"], gate=True)
            time(x + "right.", m["right"])
        else:
            attn(x + "left.", m["left"], weight=True)
            delta(x + "right.", m["right"])
            w[x + "left.out"], w[x + "right.out"] = 1.0 + 0.2 * n(H), 1.0 + 0.2 * n(H)
        for q in (1, 2) if L.get("mlp") else (1,):
            w[f"{p}hc{q}.in"], w[f"{p}hc{q}.out"], w[f"{p}hc{q}.mix"] = u(0.4, 1.2, S), u(0.5, 1.3, S), torch.eye(S) * 0.9 + 0.15 * n(S, S)
        if L.get("mlp"):
            norm(p + "norm2")
            z, E, f = p + "mlp.", L["mlp"]["router"]["experts"], L["mlp"]["expert"]["ff"]
            w[z + "router"] = 1.5 * lin(E, H)
            if not close_calls:
                b = w[p + "norm2.b"]
                w[z + "router"] = 0.1 * lin(E, H) + (torch.randperm(E, generator=g).float() - E / 2)[:, None] * b / b.square().sum()
            for j in range(E):
                w[z + f"e{j}.up"], w[z + f"e{j}.down"] = lin(f, H), lin(H, f)
    return w


def att(heads, kv_heads, dim, vdim, chunk, reach, mlp=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or round(2.0 / dim ** 0.5, 4), "bias_max": reach, "mask": {"size": chunk}}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def left(heads, kv_heads, dim, vdim, rot, base=10000.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": round(1.6 / dim ** 0.5, 4), "rot": {"base": base, "dims": rot}}


def par(lft, heads, dim, scales=(0.8, 1.2), mlp=None):
    return {"type": "parallel", "mixer": {"left": lft, "right": {"heads": heads, "dim": dim}, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def par2(lft, heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "parallel_2", "mixer": {"left": lft, "right": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}, "mlp": mlp}


def moe_spec(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def model_cfg(width, vocab, streams, layers, eps=1e-5, mult=0.9):
    return {"architecture": "Fasodra", "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "streams": streams, "vocab": vocab, "width": width}


# several geometries: every kind first and last, layers without a feed-forward, sizes off the kernels' tiles and on them, sizes of one, key heads wider
# than the chunked recurrences and the tensor-core attention take, one stream and many
MODELS = {
    "odd": lambda: model_cfg(136, 301, 3, [att(6, 2, 24, 40, 21, 50, moe_spec(5, 2, 40)), par(left(4, 2, 20, 12, 6, 500.0), 5, 12, mlp=moe_spec(7, 3, 24)),
                                           par2(left(3, 3, 36, 20, 36), 4, 2, 24, 20, 3, moe_spec(4, 1, 56)), att(3, 1, 40, 9, 70, 20),
                                           par(left(5, 1, 9, 24, 8, 77.0), 3, 40, (-0.6, 0.5)), par2(left(2, 1, 44, 30, 10), 6, 1, 40, 12, 5)], 3e-3, 0.7),
    "tiles": lambda: model_cfg(384, 520, 2, [par2(left(4, 4, 128, 128, 64, 1e6), 4, 4, 128, 128, 4, moe_spec(12, 4, 128)), att(16, 2, 128, 64, 130, 128, moe_spec(12, 4, 128)),
                                             par(left(8, 2, 64, 64, 32), 4, 64, mlp=moe_spec(12, 4, 256)), att(8, 1, 96, 32, 64, 40, moe_spec(8, 3, 128))]),
    "ones": lambda: model_cfg(48, 40, 1, [par(left(1, 1, 2, 1, 2), 1, 1, (1.0, 1.0), moe_spec(1, 1, 1)), att(1, 1, 1, 2, 1, 9), par2(left(16, 1, 3, 1, 2, 3.0), 3, 3, 1, 1, 1, moe_spec(3, 3, 8)),
                                          att(2, 2, 8, 8, 3, 17)], 1e-6, 1.0),
    "wide": lambda: model_cfg(250, 200, 5, [att(33, 1, 24, 16, 90, 60, moe_spec(4, 1, 96)), par(left(2, 2, 200, 136, 100), 2, 160, mlp=moe_spec(6, 2, 64)),
                                            par2(left(5, 1, 260, 24, 130), 2, 1, 160, 72, 4), par2(left(2, 2, 16, 272, 16), 2, 2, 48, 200, 2, moe_spec(6, 5, 32)),
                                            par(left(70, 1, 8, 8, 4), 1, 128)], 1e-4, 1.1),
}
