"""Plain evaluation of the Rubasun design, one function per mechanism, used as the oracle of the device path.

Whole sequences at a time, keys and values written out per head, from a ``config.json`` dictionary and a dictionary of tensors under the
checkpoint's own names, in the type of the tensors.  No code is shared with the package.
"""
from __future__ import annotations

import math

import torch


def dyt(x, alpha, w, b):
    """Dynamic tanh: an element-wise stand-in for a norm, b + w tanh(alpha x)."""
    return b + w * torch.tanh(alpha * x)


def rms_norm(x, w, eps):
    return w * x * torch.rsqrt(x.square().mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh((2 / math.pi) ** 0.5 * (z + 0.044715 * z ** 3)))


def rotate(x, positions, base):
    """Rotary embedding of x [T, ..., 2n]: channels (2i, 2i + 1) turn by position * base^(-i / n)."""
    n = x.shape[-1] // 2
    f = torch.tensor([base ** (-i / n) for i in range(n)], dtype=torch.float64)
    a = positions.to(torch.float64).reshape(-1, *([1] * (x.dim() - 1))) * f
    z = torch.view_as_complex(x.to(torch.float64).reshape(*x.shape[:-1], n, 2).contiguous())
    return torch.view_as_real(z * torch.polar(torch.ones_like(a), a)).reshape(x.shape).to(x.dtype)


def latent_keys(spec, w, p, h, eps):
    """(latents [T, rank] after their norm, rotated key part [T, rot]) of a layer that makes its own."""
    y = h @ w[p + "dkv"].T
    r = spec["kv_rank"]
    return rms_norm(y[:, :r], w[p + "dkv.norm"], eps), rotate(y[:, r:], torch.arange(len(h)), spec["rot"]["base"])


def causal_attention(q, k, v, scale):
    """q, k [T, H, d], v [T, H, e] -> [T, H, e]."""
    T = len(q)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s + torch.full((T, T), float("-inf"), dtype=s.dtype).triu(1)
    return torch.einsum("hij,jhe->ihe", torch.softmax(s, -1), v)


def latent_mixer(spec, w, p, h, latents):
    """The mixer's output from its input ``h`` and the (latents, rotated key part) it attends over."""
    T, H, d, r, e = len(h), spec["heads"], spec["dim"], spec["rot_dim"], spec["vdim"]
    c, kr = latents
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    q = torch.cat([q[..., :d], rotate(q[..., d:], torch.arange(T), spec["rot"]["base"])], -1)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, d), kr[:, None, :].expand(T, H, r)], -1)
    o = causal_attention(q, k, (c @ w[p + "uv"].T).view(T, H, e), spec["scale"])
    return (o * torch.sigmoid(h @ w[p + "g"].T)[..., None]).reshape(T, H * e) @ w[p + "o"].T


def dense_ff(w, p, h):
    return (torch.nn.functional.silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(w, p, x, limit):
    """Clamped GLU with a steeper sigmoid and a shifted linear half."""
    g = torch.clamp(x @ w[p + "gate"].T, max=limit)
    u = torch.clamp(x @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def route(logits, top):
    """(ids, weights) [T, top]: sigmoid scores, the largest ones, as they are."""
    s = torch.sigmoid(logits)
    return s.topk(top, dim=-1).indices, s.topk(top, dim=-1).values


def moe(spec, w, p, h):
    ids, wt = route(h @ w[p + "router"].T, spec["router"]["top"])
    y = torch.zeros_like(h)
    for t in range(len(h)):
        for i, c in zip(ids[t].tolist(), wt[t]):
            y[t] += expert(w, p + f"e{i}.", (c * h[t])[None], spec["expert"]["limit"])[0]
    sh = spec.get("shared")
    if sh:
        y = y + torch.sigmoid(h @ w[p + "shared.sg"].T) * expert(w, p + "shared.", h, sh["limit"])
    return y


def token_side(w, p, x, e, eps):
    """The update that a layer takes from its own slice ``e`` of the token table."""
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return rms_norm(y, w[p + "norm"], eps)


def forward(cfg, w, tokens, want_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer)."""
    eps = cfg["norm"]["eps"]
    ids = torch.as_tensor(tokens)
    nrm = lambda x, n: dyt(x, w[n + ".alpha"], w[n], w[n + ".b"])
    x = w["embed"][ids] * cfg["embedding"]["scale"]
    side = (cfg.get("token_side") or {}).get("dim", 0)
    held, layers = {}, []
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = nrm(x, p + "norm1")
        src = m.get("kv_from")
        held[i] = latent_keys(m, w, p + "mix.", h, eps) if src is None else held[src]
        x = x + nrm(latent_mixer(m, w, p + "mix.", h, held[i]), p + "norm1b")
        if L.get("mlp"):
            h = nrm(x, p + "norm2")
            y = dense_ff(w, p + "mlp.", h) if L["mlp"]["kind"] == "dense" else moe(L["mlp"], w, p + "mlp.", h)
            x = x + nrm(y, p + "norm2b")
        if side:
            x = x + token_side(w, p + "side.", x, w["side.embed"][ids][:, i * side: (i + 1) * side], eps)
        layers.append(x)
    lg = nrm(x, "final.norm") @ w["head"].T
    return (lg, layers) if want_layers else lg


# ------------------------------------------------------------------------------------------------ random models
def random_model(cfg, seed=0, sharp=1.0, close_calls=True):
    """Tensors for a configuration, spread so that every mechanism matters.  ``sharp`` scales the queries: large values make single keys stand
    out of the softmax.  Without ``close_calls`` the bias of the norm in front of a router decides the choice (rounding cannot turn it)."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    u = lambda lo, hi, *s: lo + (hi - lo) * torch.rand(s, generator=g)
    H, V, w = cfg["width"], cfg["vocab"], {}
    lin = lambda o, i: n(o, i) / i ** 0.5
    side = (cfg.get("token_side") or {}).get("dim", 0)

    def norm(p):
        w[p], w[p + ".b"], w[p + ".alpha"] = 1.0 + 0.2 * n(H), 0.3 * n(H), u(0.4, 1.2)

    def unit(p, f):
        w[p + "gate"], w[p + "up"], w[p + "down"] = 1.5 * lin(f, H), 1.5 * lin(f, H), lin(H, f)

    w["embed"], w["head"] = n(V, H), lin(V, H)
    norm("final.norm")
    if side:
        w["side.embed"] = n(V, side * len(cfg["layers"]))
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        x, h, d, r, e, c = p + "mix.", m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        norm(p + "norm1")
        norm(p + "norm1b")
        w[x + "q"], w[x + "uk"], w[x + "uv"], w[x + "g"], w[x + "o"] = sharp * lin(h * (d + r), H), lin(h * d, c), lin(h * e, c), lin(h, H), lin(H, h * e)
        if m.get("kv_from") is None:
            w[x + "dkv"], w[x + "dkv.norm"] = lin(c + r, H), 1.0 + 0.2 * n(c)
        if L.get("mlp"):
            norm(p + "norm2")
            norm(p + "norm2b")
            z = p + "mlp."
            if L["mlp"]["kind"] == "dense":
                unit(z, L["mlp"]["ff"])
            else:
                E = L["mlp"]["router"]["experts"]
                w[z + "router"] = 1.5 * lin(E, H)
                if not close_calls:
                    b = w[p + "norm2.b"]
                    w[z + "router"] = 0.1 * lin(E, H) + (torch.randperm(E, generator=g).float() - E / 2)[:, None] * b / b.square().sum()
                for j in range(E):
                    unit(z + f"e{j}.", L["mlp"]["expert"]["ff"])
                if L["mlp"].get("shared"):
                    unit(z + "shared.", L["mlp"]["shared"]["ff"])
                    w[z + "shared.sg"] = lin(1, H)
        if side:
            w[p + "side.gate"], w[p + "side.proj"], w[p + "side.norm"] = lin(side, H), lin(H, side), 0.5 * (1.0 + 0.2 * n(H))
    return w


def lat(heads, dim, rot_dim, vdim, kv_rank, kv_from=None, mlp=None, base=10000.0, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": {"base": base, "dims": rot_dim},
         "scale": scale or round(1.3 / (dim + rot_dim) ** 0.5, 4)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe_spec(experts, top, ff, limit=1.5, shared=0, shared_limit=2.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top},
            "shared": {"ff": shared, "limit": shared_limit} if shared else None}


def model_cfg(width, vocab, layers, eps=1e-5, scale=1.5, side=0):
    return {"architecture": "Rubasun", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "token_side": {"dim": side} if side else None,
            "vocab": vocab, "width": width}


# several geometries: rows shared forwards and past layers with their own, layers without a feed-forward, sizes off the kernels' tiles and on them,
# sizes of one, latents wider than the tensor-core kernel takes, models without a side table or a shared expert
MODELS = {
    "odd": lambda: model_cfg(136, 301, [lat(6, 24, 10, 20, 40, mlp=dense(104)), lat(6, 20, 12, 24, 56, mlp=moe_spec(5, 2, 40, shared=72), base=500.0),
                                        lat(3, 36, 10, 9, 40, 0), lat(10, 12, 12, 16, 56, 1, moe_spec(7, 3, 24, 0.7, 40, 0.5), base=500.0),
                                        lat(2, 44, 6, 30, 24, mlp=dense(60), base=77.0)], 3e-2, 0.8, 13),
    "tiles": lambda: model_cfg(384, 520, [lat(20, 128, 64, 128, 512, mlp=dense(512)), lat(12, 64, 64, 64, 512, 0, moe_spec(12, 4, 128, shared=256)),
                                          lat(40, 64, 32, 64, 256, mlp=moe_spec(8, 2, 256, 3.0, 128, 1.0), base=1e5), lat(8, 96, 32, 128, 256, 2, base=1e5)], 1e-5, 2.0, 64),
    "ones": lambda: model_cfg(48, 40, [lat(1, 1, 2, 1, 1, mlp=moe_spec(1, 1, 1, shared=1)), lat(1, 8, 2, 8, 8, mlp=moe_spec(3, 3, 8, 2.0)), lat(16, 1, 2, 3, 1, 0, dense(1))],
                              1e-6, 1.0, 1),
    "wide": lambda: model_cfg(250, 200, [lat(33, 24, 16, 16, 600, mlp=moe_spec(4, 1, 96, 1.0)), lat(5, 200, 16, 136, 600, 0, dense(136), scale=0.05),
                                         lat(70, 8, 8, 8, 128, mlp=moe_spec(6, 2, 64, 0.6, 200))], 1e-4, 3.0),
}
