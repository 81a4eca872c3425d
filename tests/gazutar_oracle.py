"""Plain fp32 / fp64 evaluation of the Gazutar design, one function per mechanism, used as the oracle of the device path.

Everything works on whole sequences, token by token where the mechanism is a recurrence, from a ``config.json`` dictionary and a
dictionary of tensors under the checkpoint's own names.  No code is shared with the package.
"""
from __future__ import annotations

import json
import math
import struct

import torch

UNIT_EPS = 1e-6           # inside the square root of the recurrent layers' unit vectors


def layer_norm(x, w, b, eps):
    mu = x.mean(-1, keepdim=True)
    d = x - mu
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def slopes(n_heads, dtype=torch.float32):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / n_heads) for h in range(n_heads)], dtype=dtype)


def windowed_attention(q, k, v, scale, window, slope):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e].  Softmax over 0 <= i - j < window (0: the whole prefix) of
    scale q.k - slope_h (i - j)."""
    T, H, _ = q.shape
    G = k.shape[1]
    kk, vv = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    dist = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    s = s - slope[:, None, None] * dist.to(q.dtype)
    seen = (dist >= 0) & ((dist < window) if window else torch.ones_like(dist, dtype=torch.bool))
    s = s.masked_fill(~seen, float("-inf"))
    return torch.einsum("hij,jhe->ihe", torch.softmax(s, -1), vv)


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention_mixer(spec, eps, w, p, h, v_first):
    """Returns (output, this layer's own values before mixing)."""
    T = h.shape[0]
    H, G, d, e = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).view(T, H, d)
    k = rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).view(T, G, d)
    v = h @ w[p + "v"].T
    own = v
    if spec.get("v_mix") and v_first is not None:
        v = mix_values(v, v_first, w[p + "vmix"])
    window = (spec.get("mask") or {}).get("size", 0)
    o = windowed_attention(q, k, v.view(T, G, e), spec["scale"], window, slopes(H, h.dtype)).reshape(T, H * e)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T, own


def short_conv(x, taps):
    """x [T, C], taps [C, n]: causal, last column = current token; then SiLU."""
    n = taps.shape[1]
    xp = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x])
    y = sum(xp[j: j + x.shape[0]] * taps[:, j] for j in range(n))
    return y * torch.sigmoid(y)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def delta_rule(q, k, v, g, beta, S=None):
    """q, k, g [T, H, d], v [T, H, e], beta [T, H] -> ([T, H, e], state [H, d, e]); decay, read, write, read out."""
    T, H, d = q.shape
    e = v.shape[2]
    S = torch.zeros(H, d, e, dtype=q.dtype) if S is None else S
    out = torch.empty(T, H, e, dtype=q.dtype)
    for t in range(T):
        S = S * g[t][:, :, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hde,hd->he", S, q[t])
    return out, S


def delta_mixer(spec, eps, w, p, h):
    T = h.shape[0]
    H, G, d, e = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q, k, v = (short_conv(h @ w[p + n].T, w[p + n + ".conv"]) for n in ("q", "k", "v"))
    q = unit(q.view(T, G, d)) * d ** -0.5
    k = unit(k.view(T, G, d))
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    a = ((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).view(T, H, d)
    g = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(a))
    o, _ = delta_rule(q, k, v.view(T, H, e), g, beta)
    o = rms_norm(o, w[p + "norm"], eps)
    gate = torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return (o.reshape(T, H * e) * gate) @ w[p + "o"].T


def route(router, s_logits, correction):
    """Choice of one token batch: (ids [T, top], weights [T, top]) from router logits."""
    s = torch.softmax(s_logits, -1)
    choice = s + correction
    g = router.get("groups")
    T, n = s.shape
    if g and g["count"] > 1:
        per = n // g["count"]
        best = choice.view(T, g["count"], per).max(-1).values
        keep = torch.zeros_like(best, dtype=torch.bool).scatter_(1, best.topk(g["keep"], dim=1).indices, True)
        choice = choice.masked_fill(~keep.repeat_interleave(per, 1), float("-inf"))
    ids = choice.topk(router["top"], dim=1).indices
    return ids, s.gather(1, ids)


def expert(w, p, x):
    z = x @ w[p + "gate"].T
    return (z * torch.sigmoid(z) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def moe(spec, w, p, h):
    r = spec["router"]
    ids, wt = route(r, h @ w[p + "router"].T, w[p + "correction"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for i, c in zip(ids[t].tolist(), wt[t]):
            y[t] += c * (h[t] if i >= r["experts"] else expert(w, p + f"e{i}.", h[t: t + 1])[0])
    return y


def forward(cfg, w, tokens, want_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer)."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    layers, v_first = [], None
    for i, spec in enumerate(cfg["layers"]):
        p = f"l{i}."
        if spec["type"] == "attention":
            y, own = attention_mixer(spec["mixer"], eps, w, p + "mix.", x, v_first)
            if spec["mixer"].get("v_mix") and v_first is None:
                v_first = own
        else:
            y = delta_mixer(spec["mixer"], eps, w, p + "mix.", x)
        x = x + layer_norm(y, w[p + "norm1"], w[p + "norm1.b"], eps)
        if spec.get("mlp"):
            x = x + layer_norm(moe(spec["mlp"], w, p + "mlp.", x), w[p + "norm2"], w[p + "norm2.b"], eps)
        layers.append(x)
    lg = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T * cfg["logit_scale"]
    return (lg, layers) if want_layers else lg


# ------------------------------------------------------------------------------------------------ files
def save_model(path, cfg, w):
    """config.json + model.safetensors (bfloat16) in ``path``; returns the tensors as the file holds them (fp32)."""
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    head, blobs, off, held = {}, [], 0, {}
    for k, t in w.items():
        b16 = t.to(torch.bfloat16).contiguous()
        held[k] = b16.float()
        raw = b16.reshape(-1).view(torch.uint8).numpy().tobytes()
        head[k] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    hj = json.dumps(head).encode()
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))
    return held


# ------------------------------------------------------------------------------------------------ random models
def random_model(cfg, seed=0, rank=20, sharp=1.0, close_calls=True):
    """Tensors for a configuration, spread so that every mechanism matters.  ``sharp`` scales the query norms: large values make single
    keys stand out of the softmax.  Without ``close_calls`` the router's correction decides the choice alone (rounding cannot turn it)."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    u = lambda lo, hi, *s: lo + (hi - lo) * torch.rand(s, generator=g)
    H, V, w = cfg["width"], cfg["vocab"], {}
    lin = lambda o, i: n(o, i) / i ** 0.5

    def ln(p):
        w[p], w[p + ".b"] = 1.0 + 0.2 * n(H), 0.2 * n(H)

    w["embed"], w["head"] = n(V, H), lin(V, H)
    ln("final.norm")
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        x = p + "mix."
        ln(p + "norm1")
        h, k, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        if L["type"] == "attention":
            w[x + "q"], w[x + "k"], w[x + "v"], w[x + "g"], w[x + "o"] = lin(h * d, H), lin(k * d, H), lin(k * e, H), lin(h * e, H), lin(H, h * e)
            w[x + "q.norm"], w[x + "k.norm"] = sharp * (1.0 + 0.2 * n(h * d)), 1.0 + 0.2 * n(k * d)
            if m.get("v_mix"):
                w[x + "vmix"] = u(0.3, 0.7)
        else:
            w[x + "q"], w[x + "k"], w[x + "v"], w[x + "b"], w[x + "o"] = lin(k * d, H), lin(k * d, H), lin(h * e, H), lin(h, H), lin(H, h * e)
            for t, c in (("q", k * d), ("k", k * d), ("v", h * e)):
                w[x + t + ".conv"] = u(-1.0, 1.0, c, m["conv"])
            w[x + "A_log"], w[x + "dt_bias"], w[x + "norm"] = u(-3.0, 0.5, h), u(-3.0, 0.0, h * d), 1.0 + 0.2 * n(e)
            w[x + "a1"], w[x + "a2"], w[x + "g1"], w[x + "g2"] = lin(rank, H), lin(h * d, rank), lin(rank + 3, H), lin(h * e, rank + 3)
        if L.get("mlp"):
            ln(p + "norm2")
            r, f = L["mlp"]["router"], L["mlp"]["expert"]["ff"]
            z = p + "mlp."
            tot = r["experts"] + (r.get("identity") or 0)
            w[z + "router"], w[z + "correction"] = 1.5 * lin(tot, H), -1.5 + 0.3 * n(tot)
            if not close_calls:
                w[z + "correction"] = 2.0 * torch.randperm(tot, generator=g).float() - tot
            for j in range(r["experts"]):
                w[z + f"e{j}.gate"], w[z + f"e{j}.up"], w[z + f"e{j}.down"] = lin(f, H), lin(f, H), lin(H, f)
    return w


def att(heads, kv_heads, dim, vdim, window=0, v_mix=False, scale=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or round(1.7 / dim ** 0.5, 4), "v_mix": v_mix}
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def moe_spec(experts, identity, top, count=1, keep=1, ff=40):
    r = {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}
    if identity:
        r["identity"] = identity
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def model_cfg(width, vocab, layers, eps=1e-5, logit_scale=0.5):
    return {"architecture": "Gazutar", "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# several geometries: unequal layers, layers without a feed-forward, groups of one head, sizes off the kernels' tiles and on them
MODELS = {
    "odd": lambda: model_cfg(136, 301, [delta(6, 2, 24, 40, 3, moe_spec(5, 1, 2, 3, 2, 40)), att(6, 2, 24, 40, 21, True, mlp=moe_spec(7, 0, 3, 1, 1, 24)),
                                        delta(2, 1, 40, 20, 5), att(4, 4, 36, 40, 9, False), att(4, 2, 20, 40, 33, True, mlp=moe_spec(4, 4, 4, 2, 1, 56))], 3e-4, 0.3),
    "attention first": lambda: model_cfg(96, 128, [att(3, 1, 32, 32, 50, True, mlp=moe_spec(6, 2, 1, 4, 2, 48)), delta(1, 1, 16, 16, 1, moe_spec(6, 2, 2, 2, 1, 48)),
                                                   att(3, 1, 16, 32, 0, True), delta(5, 5, 64, 48, 2)], 1e-6, 1.0),
    "tiles": lambda: model_cfg(384, 520, [delta(3, 3, 128, 128, 4, moe_spec(12, 4, 4, 4, 2, 128)), att(16, 1, 128, 64, 130, True, mlp=moe_spec(12, 4, 4, 4, 2, 128)),
                                          delta(4, 2, 64, 96, 4, moe_spec(12, 4, 4, 4, 2, 128)), att(8, 2, 64, 32, 70, True)], 1e-5, 0.25),
    "narrow": lambda: model_cfg(100, 67, [att(5, 5, 8, 8, 3, True, mlp=moe_spec(3, 2, 5, 5, 5, 12)), delta(5, 5, 8, 12, 7, moe_spec(3, 2, 2, 5, 4, 12)),
                                          att(10, 5, 16, 8, 1, True), delta(4, 1, 20, 8, 4)], 1e-4, 0.7),
    "wide": lambda: model_cfg(256, 200, [delta(2, 1, 160, 160, 4), att(20, 1, 192, 256, 65, True, mlp=moe_spec(3, 3, 2, 1, 1, 64)), delta(2, 2, 48, 200, 4),
                                         att(2, 2, 260, 24, 40, False)], 1e-5, 2.0),
}
