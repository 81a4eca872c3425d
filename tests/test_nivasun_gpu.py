"""Nivasun on the device against the plain evaluation in nivasun_oracle.py: every mechanism alone, then whole models of several geometries through
the engine - prompts, decoding, portions, mixed batches, reused pages and slots, generation through the server's scheduler."""
import pytest
import torch

pytestmark = pytest.mark.gpu

import nivasun_oracle as O
from gazutar_oracle import save_model
from layerstorm_b200.models.block_model import BlockModel
from layerstorm_b200.models.checkpoint import open_checkpoint
from layerstorm_b200.ops import _native as nat
from layerstorm_b200.runtime.engine import Engine, Portion

DEV = "cuda"
F32, B16, I32 = torch.float32, torch.bfloat16, torch.int32


def i32(x):
    return torch.tensor(x, dtype=I32, device=DEV)


def err(a, b):
    a, b = a.float().cpu(), b.float().cpu()
    return float((a - b).abs().max() / (b.abs().max() + 1e-12))


def exactly(t, f32):
    return t if f32 else t.to(B16).float()


def dev(t):
    return None if t is None else t.float().to(DEV).contiguous()


def steps_of(parts):
    """Staging arrays of a step of (sequence, first position, rows) parts: row_seq, row_pos, seq_row0, seq_nrows, rows per part."""
    n = [c for _, _, c in parts]
    return (i32([s for s, _, c in parts for _ in range(c)]), i32([p + j for _, p, c in parts for j in range(c)]), i32([sum(n[:j]) for j in range(len(n))]), i32(n), n)


# ------------------------------------------------------------------------------------------------ attention with shared keys and values, differential attention
def unrotate(x, pos, base, dims, pairs):
    """Rows of x [n, H, d] turned back by their positions."""
    y = x.clone()
    f = torch.tensor([base ** (-2 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = torch.as_tensor(pos, dtype=torch.float64)[:, None, None] * f
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    one, two = (slice(0, dims, 2), slice(1, dims, 2)) if pairs else (slice(0, dims // 2), slice(dims // 2, dims))
    u, v = x[..., one], x[..., two]
    y[..., one], y[..., two] = u * c + v * s, v * c - u * s
    return y


class Paged:
    """Sequences laid out over shuffled cache pages; rows of a step = runs of tokens of some of them."""

    def __init__(self, H, G, dk, dv, page, lens, f32, maps=1, seed=0):
        self.H, self.G, self.dk, self.dv, self.page, self.f32, self.maps = H, G, dk, dv, page, f32, maps
        self.dkp, self.dvp = nat.call("lsb_attn_head_pad", dk), nat.call("lsb_attn_head_pad", dv)
        g = torch.Generator().manual_seed(seed)
        self.max_pages = max((n + page - 1) // page for n in lens)
        n_pages = len(lens) * self.max_pages + 3
        self.bt = torch.randperm(n_pages, generator=g)[: len(lens) * self.max_pages].view(len(lens), -1).int().to(DEV)
        self.dt = F32 if f32 else B16
        self.cache = torch.full((n_pages, page, G * (maps * self.dkp + self.dvp)), 7.5, dtype=self.dt, device=DEV)     # stale values everywhere

    def run(self, parts, window, scale, rot, base, NS=1, temp=None, sink=None, lam=0.0, eps=1e-5, factor=1.0):
        """parts: (sequence, first position, q [n, H maps dk], k [n, G maps dk], v [n, G dv] or None: the keys)."""
        H, G, dk, dv, M = self.H, self.G, self.dk, self.dv, self.maps
        shared = parts[0][4] is None
        proj = torch.cat([torch.cat(p[2:4] if shared else p[2:], 1) for p in parts]).float().to(DEV).contiguous()
        seq, pos, row0, nrows, n = steps_of([(p[0], p[1], len(p[2])) for p in parts])
        R = proj.shape[0]
        q = torch.zeros(R, H * M, self.dkp, dtype=self.dt, device=DEV)
        out = torch.full((R, H * dv + 8), 3.0, dtype=self.dt, device=DEV)
        op, ml = torch.full((R * H * M * NS * self.dvp,), float("nan"), device=DEV), torch.full((R * H * M * NS * 2,), float("nan"), device=DEV)
        inv = torch.tensor([base ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float64, device=DEV)
        ok = H * M * dk
        nat.call("lsb_attn_head_prep", proj, proj.shape[1], 0, ok, ok if shared else ok + G * M * dk, None, None, None, 0, None, None, 1e-5, rot, int(M > 1), inv, dev(temp), M, q,
                 self.cache, self.bt, self.max_pages, seq, pos, R, H * M, G * M, dk, dv, self.dkp, self.dvp, self.page, int(self.f32))
        nat.call("lsb_attn", q, self.cache, self.bt, self.max_pages, self.page, seq, pos, row0, nrows, len(n), max(n), proj, proj.shape[1], -1, out, H * dv + 8, op, ml, NS, R,
                 H * M, G * M, dk, dv, self.dkp, self.dvp, window, scale, None, 0, 0, None, 0, 1.0, dev(sink), M, int(self.f32))
        if M > 1:
            k = nat.call("lsb_attn_partials", max(n), H * M, G * M, self.dkp, self.dvp, NS, int(self.f32))
            nat.call("lsb_attn_diff", out, H * dv + 8, op, ml, k, R, H, H // G, dv, self.dvp, lam, eps, factor, seq, int(self.f32))
        torch.cuda.synchronize()
        assert float((out[:, H * dv:].float() - 3.0).abs().max()) == 0
        return out[:, : H * dv].float().cpu()


def spots(i, window, page):
    """Positions that a query at i may be made to look at: itself, the last visible key, the one just outside, page borders, the token in front, the first."""
    return [max(0, min(i, j)) for j in (i, i - window + 1, i - window, i // page * page, i // page * page - 1, i - 1, 0)]


def schedules(P, run, ref, data, lens, tol, window):
    """A prompt and the first tokens of another, portions, single rows with and without key splits, runs of two, portions of 19."""
    top = max(float(r.abs().max()) for r in ref)                     # rows that a sink empties are held against the others
    off = lambda a, b: float((a.float() - b).abs().max()) / top
    cut = lambda s, a, z: (s, a, *(None if t is None else t[a:z] for t in data[s]))
    T = lens[0]
    p = P(0)
    out = run(p, [cut(0, 0, T), cut(1, 0, 3)], 1)
    assert off(out, torch.cat([ref[0], ref[1][:3]])) < tol
    assert off(run(p, [cut(1, 3, 70)], 1), ref[1][3:70]) < tol
    for a in range(70, lens[1]):                                     # decoded
        for NS in ((1, 3) if a % 10 == 0 or a % window < 2 else (1,)):
            assert off(run(p, [cut(1, a, a + 1)], NS), ref[1][a: a + 1]) < tol, (a, NS)
    p = P(9)
    outs = [run(p, [cut(0, a, a + 2), cut(1, a, a + 2)], 1 + a // 2 % 2) for a in range(0, 120, 2)]
    assert off(torch.cat([o[:2] for o in outs]), ref[0][:120]) < tol and off(torch.cat([o[2:] for o in outs]), ref[1][:120]) < tol
    p = P(5)
    assert off(torch.cat([run(p, [cut(0, a, min(T, a + 19))], 2) for a in range(0, T, 19)]), ref[0]) < tol


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,G,dk,rot,window", [(4, 2, 32, 32, 37), (6, 1, 24, 10, 21), (8, 8, 64, 64, 64), (3, 3, 96, 96, 50), (20, 1, 128, 64, 33), (2, 1, 200, 100, 48), (2, 2, 272, 272, 40),
                                               (33, 1, 40, 8, 100), (1, 1, 2, 2, 1), (5, 5, 20, 20, 500)])
def test_windowed_attention_over_shared_keys_with_sinks_and_temperatures(H, G, dk, rot, window, f32):
    """One key stands out for every query: at the window's ends, just outside (then only the sink and the rest are left), at page borders.  Sinks lie between
    the scores and far above them, temperatures differ per head; the values are the keys in front of their rotation."""
    if f32 and (H, G) not in ((6, 1), (3, 3)):
        pytest.skip("the CUDA-core kernel has one form")
    T, page, base = 150, 16, 300.0
    g = torch.Generator().manual_seed(H * 100 + dk)
    temp = 0.5 + torch.rand(H, generator=g) * 1.5
    sink = torch.where(torch.arange(H) % 3 == 2, 14.0, 3.0 * torch.randn(H, generator=g))
    lens, data = [T, T - 29], []
    for n in lens:
        k = torch.nn.functional.normalize(torch.randn(n, G, dk, generator=g), dim=-1) * dk ** 0.5
        kr, q = O.rotate_half(k, rot, base), torch.empty(n, H, dk)
        for i in range(n):
            for h in range(H):
                q[i, h] = 11.0 / dk * kr[spots(i, window, page)[(i + h) % 7], h // (H // G)]
        q = unrotate(q, range(n), base, rot, False)
        data.append((exactly(q.reshape(n, -1), f32), exactly(k.reshape(n, -1), f32), None))
    ref = []
    for q, k, _ in data:
        q, k = q.view(-1, H, dk), k.view(-1, G, dk)
        ref.append(O.attend(O.rotate_half(q, rot, base), O.rotate_half(k, rot, base), k, 0.9, window, temp, sink).flatten(1))
    schedules(lambda seed: Paged(H, G, dk, dk, page, lens, f32, seed=seed), lambda p, parts, NS: p.run(parts, window, 0.9, rot, base, NS, temp, sink), ref, data, lens,
              2e-5 if f32 else 1.2e-2, window)


def test_a_sink_counts_once_and_takes_no_part_in_the_values():
    """A first token alone: its weight is e^s / (e^s + e^sink), whatever the form, and vanishes under a huge sink without an overflow."""
    for f32 in (True, False):
        for sink in (-200.0, -1.0, 2.5, 200.0):
            for n in (1, 9):
                q, k = torch.ones(n, 32), torch.ones(n, 32) * 0.25
                P = Paged(1, 1, 32, 32, 16, [32], f32)
                o = P.run([(0, 0, q, k, None)], 1, 0.125, 2, 10.0, sink=torch.tensor([sink]))[0, 0]
                w = 1.0 / (1.0 + torch.exp(torch.tensor(sink - 1.0)))
                assert abs(float(o) - 0.25 * float(w)) < (1e-6 if f32 else 2e-3), (f32, sink, n)


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,G,dk,dv,rot,window", [(4, 4, 48, 64, 16, 37), (6, 3, 20, 36, 12, 26), (8, 2, 64, 128, 64, 64), (4, 1, 128, 128, 128, 33), (2, 1, 264, 72, 100, 41), (5, 5, 16, 280, 10, 64),
                                                  (40, 1, 24, 16, 24, 90), (1, 1, 2, 1, 2, 1), (3, 3, 96, 256, 32, 500), (4, 2, 200, 250, 64, 45)])
def test_differential_attention_forms(H, G, dk, dv, rot, window, f32):
    """The two maps of a head look at different keys, at the window's ends and page borders, over one set of values."""
    if f32 and (H, G) not in ((6, 3), (4, 1)):
        pytest.skip("the CUDA-core kernel has one form")
    T, page, base, lam, diff, eps = 150, 16, 200.0, 0.63, 0.35, 1e-4
    g = torch.Generator().manual_seed(H * 100 + dk)
    lens, data = [T, T - 29], []
    for n in lens:
        k = torch.nn.functional.normalize(torch.randn(n, 2 * G, dk, generator=g), dim=-1) * dk ** 0.5
        kr, q = O.rotate_pairs(k, rot, base), torch.empty(n, 2 * H, dk)
        for i in range(n):
            for j in range(2 * H):
                q[i, j] = 8.0 / dk * kr[spots(i, window, page)[(i + j) % 7], j // 2 // (H // G) * 2 + j % 2]
        q = unrotate(q, range(n), base, rot, True)
        data.append(tuple(exactly(t.reshape(n, -1), f32) for t in (q, k, torch.randn(n, G, dv, generator=g))))
    ref = []
    for q, k, v in data:
        q, k, v = O.rotate_pairs(q.view(-1, H, 2, dk).flatten(1, 2), rot, base).unflatten(1, (H, 2)), O.rotate_pairs(k.view(-1, 2 * G, dk), rot, base).unflatten(1, (G, 2)), v.view(-1, G, dv)
        a = [O.attend(q[:, :, i], k[:, :, i], v, 0.9, window) for i in (0, 1)]
        ref.append((O.rms(a[0] - lam * a[1], eps) * (1 - diff)).flatten(1))
    schedules(lambda seed: Paged(H, G, dk, dv, page, lens, f32, 2, seed), lambda p, parts, NS: p.run(parts, window, 0.9, rot, base, NS, lam=lam, eps=eps, factor=1 - diff), ref, data,
              lens, 1e-4 if f32 else 2.5e-2, window)


# ------------------------------------------------------------------------------------------------ latent attention without positions
class Latent:
    """A latent layer's cache over shuffled pages and its weights, as the model lays them out."""

    def __init__(self, H, dn, dv, dl, page, lens, f32, seed=0):
        self.sz, self.page, self.f32, self.dt = (H, dn, dv, dl), page, f32, F32 if f32 else B16
        self.dlp, self.dnp = nat.call("lsb_latent_pad", dl), (dn + 7) // 8 * 8
        g = torch.Generator().manual_seed(seed)
        self.max_pages = max((n + page - 1) // page for n in lens)
        n_pages = len(lens) * self.max_pages + 3
        self.bt = torch.randperm(n_pages, generator=g)[: len(lens) * self.max_pages].view(len(lens), -1).int().to(DEV)
        self.cache = torch.full((n_pages, page, self.dlp), 7.5, dtype=self.dt, device=DEV)

    def weights(self, uk, uv, kvn):
        H, dn, dv, dl = self.sz
        self.uk, self.uv = torch.zeros(H, self.dlp, self.dnp, dtype=self.dt, device=DEV), torch.zeros(H, dv, self.dlp, dtype=self.dt, device=DEV)
        self.uk[:, :dl, :dn], self.uv[:, :, :dl], self.kvn = uk.view(H, dn, dl).transpose(1, 2).to(DEV), uv.view(H, dv, dl).to(DEV), dev(kvn)
        return self

    def run(self, parts, window, scale, NS=1, eps=1e-5):
        """parts: (sequence, first position, q [n, H dn], y [n, dl], gate logits [n, H dv])."""
        H, dn, dv, dl = self.sz
        q = torch.cat([p[2] for p in parts]).float().to(DEV).contiguous()
        proj = torch.cat([torch.cat(p[3:], 1) for p in parts]).float().to(DEV).contiguous()
        seq, pos, row0, nrows, n = steps_of([(p[0], p[1], len(p[2])) for p in parts])
        R, ld = len(q), proj.shape[1]
        z = lambda *s, dt=self.dt: torch.full(s, float("nan"), dtype=dt, device=DEV)
        ldo = (H * dv + 7) // 8 * 8
        ql, qn, ol, out = z(R, H, self.dlp), z(R, H, self.dnp, dt=B16), z(R, H, self.dlp), z(R, ldo)
        op, ml, e = z(R * H * NS * self.dlp, dt=F32), z(R * H * NS * 2, dt=F32), torch.zeros(1, dtype=I32, device=DEV)
        nat.call("lsb_latent_query", q, q.shape[1], proj, ld, 0, self.kvn, eps, None, self.uk, ql, qn, self.cache, self.bt, self.max_pages, self.page, seq, pos, R, H, dn, self.dnp, 0,
                 dl, int(self.f32), e)
        nat.call("lsb_latent_attn", ql, self.cache, self.bt, self.max_pages, self.page, seq, pos, row0, nrows, len(n), max(n), proj, ld, -1, ol, op, ml, NS, R, H, dl, 0, window, scale,
                 int(self.f32))
        nat.call("lsb_latent_out", out, ldo, ol, op, ml, nat.call("lsb_latent_partials", NS), self.uv, proj, ld, dl, 0, seq, R, H, dl, dv, int(self.f32), e)
        torch.cuda.synchronize()
        assert int(e[0]) == 0
        return out[:, : H * dv].float().cpu()


def latent_case(H, dn, dv, dl, window, page, lens, f32, seed):
    """Sequences whose queries look at one cached row each: at the window's ends, just outside, at page borders."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    uk, uv, kvn = exactly(n(H * dn, dl) / dl ** 0.5, f32), exactly(n(H * dv, dl) / dl ** 0.5, f32), 1.0 + 0.1 * n(dl)
    data, ref = [], []
    for T in lens:
        y, gt = n(T, dl), n(T, H * dv)
        c = O.rms(y, 1e-5) * kvn
        k, v, q = (c @ uk.T).view(T, H, dn), (c @ uv.T).view(T, H, dv), torch.empty(T, H, dn)
        for i in range(T):
            for h in range(H):
                t = k[spots(i, window, page)[(i + h) % 7], h]
                q[i, h] = 9.0 * t / (t.square().sum() + 0.1)
        q = exactly(q.reshape(T, -1), f32)
        ref.append(O.attend(q.view(T, H, dn), k, v, 1.0, window).flatten(1) * torch.sigmoid(gt))
        data.append((q, y, gt))
    return (uk, uv, kvn), data, ref


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,dn,dv,dl,window", [(6, 64, 48, 80, 37), (5, 20, 12, 44, 33), (3, 128, 128, 512, 70), (20, 32, 24, 200, 64), (2, 24, 40, 540, 50), (1, 3, 1, 5, 1), (40, 16, 16, 64, 500)])
def test_windowed_latent_attention_with_a_gate_per_channel(H, dn, dv, dl, window, f32):
    if f32 and H not in (5, 6):
        pytest.skip("the CUDA-core kernel has one form")
    lens, page = [150, 121], 16
    (uk, uv, kvn), data, ref = latent_case(H, dn, dv, dl, window, page, lens, f32, H + dl)
    most = 8 if not f32 and dl <= 512 else 1
    sizes = {1: 1, 2: 2 if most > 1 else 1, 3: most}
    schedules(lambda seed: Latent(H, dn, dv, dl, page, lens, f32, seed).weights(uk, uv, kvn), lambda p, parts, NS: p.run(parts, window, 1.0, sizes[NS] if max(len(x[2]) for x in parts) == 1 else 1),
              ref, data, lens, 3e-5 if f32 else 3e-2, window)


@pytest.mark.parametrize("H,dn,dv,dl,window", [(6, 64, 48, 80, 37), (3, 40, 24, 200, 64), (4, 128, 128, 512, 100), (2, 24, 40, 540, 500)])
def test_long_runs_over_written_out_keys_start_at_the_first_visible_one(H, dn, dv, dl, window):
    lens, page = [260], 16
    (uk, uv, kvn), data, ref = latent_case(H, dn, dv, dl, window, page, lens, False, 3)
    dnw, dvp = (dn + 15) // 16 * 16, nat.call("lsb_attn_head_pad", dv)
    P = Latent(H, dn, dv, dl, page, lens, False).weights(uk, uv, kvn)
    w = torch.zeros(H * (dnw + dvp), P.dlp, dtype=B16, device=DEV)
    w[: H * dnw].view(H, dnw, P.dlp)[:, :dn, :dl] = uk.view(H, dn, dl).to(DEV)
    w[H * dnw:].view(H, dvp, P.dlp)[:, :dv, :dl] = uv.view(H, dv, dl).to(DEV)
    e, ldo = torch.zeros(1, dtype=I32, device=DEV), (H * dv + 7) // 8 * 8
    for a, b in ((0, 130), (130, 133), (133, 260)):
        q, proj = data[0][0][a:b].to(DEV).contiguous(), torch.cat(data[0][1:], 1)[a:b].to(DEV).contiguous()
        R, base = b - a, max(0, a - window + 1)
        Tm = (b - base + 255) // 256 * 256
        z = lambda *s: torch.full(s, float("nan"), dtype=B16, device=DEV)
        qh, latr, kv, out = z(R, H, dnw), z(Tm, P.dlp), z(Tm, H * (dnw + dvp)), z(R, ldo)
        seq, pos = i32([0] * R), i32(list(range(a, b)))
        nat.call("lsb_latent_expand", q, q.shape[1], proj, proj.shape[1], 0, P.kvn, 1e-5, None, w, qh, latr, kv, P.cache, P.bt, P.max_pages, page, seq, pos, R, base, b, Tm, H, dn, dnw, 0, dl,
                 dvp, e)
        nat.call("lsb_attn_run", qh, kv, Tm, i32([0]), seq, pos, i32([0]), i32([R]), proj, proj.shape[1], dl, 0, out, ldo, R, H, dnw, 0, dv, dvp, window, base, 1.0)
        torch.cuda.synchronize()
        assert int(e[0]) == 0 and err(out[:, : H * dv], ref[0][a:b]) < 2e-2, (a, b)


# ------------------------------------------------------------------------------------------------ input convolution, residual update, embedding, router, logits
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6, 17])
@pytest.mark.parametrize("width", [16, 136, 1024])
def test_input_convolution_across_portions(width, taps, f32):
    """Runs of every short length on interleaved slots, single rows through the residual update, against the whole sequence."""
    g = torch.Generator().manual_seed(width + taps)
    T, eps, dt = 110, 1e-5, F32 if f32 else B16
    w, nw, add = torch.randn(width, taps, generator=g), 0.5 + torch.rand(width, generator=g), torch.randn(width, generator=g)
    hs = [exactly(torch.randn(T, width, generator=g), f32) for _ in range(2)]
    ref = [h + O.input_conv(h, w) for h in hs]
    dw, tol = w.T.contiguous().to(DEV), 2e-6 if f32 else 6e-3
    state = torch.zeros(4, max(1, taps - 1), width, device=DEV)
    state[1] = 50.0
    st = state if taps > 1 else None
    at = [0, 0]
    for a, b in [(1, 2), (2, 1), (40, 16), (3, 17), (16, 33), (1, 0), (0, 1), (47, 40)]:
        parts = [(s, j, n) for s, j, n in ((2, 0, a), (0, 1, b)) if n]
        x = torch.cat([hs[j][at[j]: at[j] + n] for _, j, n in parts]).to(dt).to(DEV).contiguous()
        out, n = torch.full_like(x, float("nan")), [p[2] for p in parts]
        nat.call("lsb_input_conv", out, x, width, dw, st, taps, width, i32([sum(n[:j]) for j in range(len(n))]), i32(n), i32([p[0] for p in parts]), len(n), len(x), width, int(f32))
        r0 = 0
        for _, j, c in parts:
            assert err(out[r0: r0 + c], ref[j][at[j]: at[j] + c]) < tol, (j, at, c)
            r0, at[j] = r0 + c, at[j] + c
    assert at == [110, 110] and float((state[1] - 50.0).abs().max()) == 0 and float(state[3].abs().max()) == 0
    # one row per sequence: residual update with a pass's vector, norm and convolution in one launch, slot order reversed, one idle row
    state.zero_()
    x = [torch.randn(T, width, generator=g) for _ in range(2)]
    h = [exactly(O.rms(t + add, eps) * nw, f32) for t in x]
    ref = [t + O.input_conv(t, w) for t in h]
    for t in range(24):
        resid = torch.stack([x[1][t] * 0.25, torch.zeros(width), x[0][t] * 0.25]).to(DEV)
        sub = 3.0 * resid
        act, conv = torch.zeros(3, width, dtype=dt, device=DEV), torch.zeros(3, width, dtype=dt, device=DEV)
        nat.call("lsb_resid_update", act, width, resid, width, sub, width, 3, None, None, None, 0, dev(nw), None, None, 3, width, eps, None, None, None, None, 0, 0, 0, dev(add), conv, dw,
                 st, i32([3, -1, 0]), taps, width, int(f32))
        assert err(resid[[0, 2]], torch.stack([x[1][t], x[0][t]]) + add) < 1e-6
        assert err(act[[0, 2]], torch.stack([h[1][t], h[0][t]])) < (2e-6 if f32 else 8e-3)
        assert err(conv[[0, 2]], torch.stack([ref[1][t], ref[0][t]])) < (4e-6 if f32 else 1.5e-2), t
    assert float(state[1].abs().max()) == 0 and float(state[2].abs().max()) == 0


def test_bigram_embedding_rows():
    V, H, B, mp, mc = 50, 72, 37, 2000000011, 1999999973                      # products beyond 32 bits
    g = torch.Generator().manual_seed(1)
    e, b = torch.randn(V, H, generator=g).to(B16), torch.randn(B + 1, H, generator=g).to(B16)
    toks = torch.randint(0, V, (30,), generator=g).tolist()
    out = torch.zeros(30, H, device=DEV)
    nat.call("lsb_embedding_bigram", out, e.to(DEV), b.to(DEV), i32(toks), i32([-1] + toks[:-1]), 30, H, V, 1.75, B, mp, mc)
    c = {"embedding": {"scale": 1.75, "bigram": {"buckets": B, "mul_prev": mp, "mul_cur": mc}}}
    assert err(out, O.embed(c, {"embed": e.float(), "bigram": b.float()}, toks)) < 1e-6


def test_router_bias_is_part_of_the_logits():
    """The choice follows logit + bias and the weights are the softmax of those sums; far smaller logits still keep their order."""
    R, E, top = 40, 11, 4
    g = torch.Generator().manual_seed(1)
    lg, b = torch.randn(R, E, generator=g) * 3, 4.0 * torch.randn(E, generator=g)
    lg[0] = -400.0 * torch.arange(E)
    ids, wt = O.route(lg + b, top)
    di, dw = torch.zeros(R, top, dtype=I32, device=DEV), torch.zeros(R, top, device=DEV)
    nat.call("lsb_router_topk_grouped", lg.to(DEV), dev(b), di, dw, R, E, top, 1, 1, 3, 1, 1.0, 0, E, 1)
    assert torch.equal(di.cpu().long(), ids) and err(dw, wt) < 1e-5


def test_soft_cap_of_the_logits():
    x = torch.randn(5, 301) * 40
    d = x.to(DEV)
    nat.call("lsb_softcap", d, 301, 3, 301, 9.0)
    assert err(d[:3], 9.0 * torch.tanh(x[:3] / 9.0)) < 1e-6 and torch.equal(d[3:].cpu(), x[3:])


# ------------------------------------------------------------------------------------------------ whole models
LONG = 200
_cache = {}


def load(tmp_path_factory, name, dtype):
    """(raw config, device model, tokens, logits of the oracle) of one geometry; models are built once.  The bf16 models have no close routing
    calls: a choice that rounding turns is no error of the kernels (routing itself is checked in fp32)."""
    key = (name, dtype, "files")
    if key not in _cache:
        c = O.MODELS[name]()
        d = tmp_path_factory.mktemp("nivasun")
        w = save_model(d, c, O.random_model(c, 11, close_calls=dtype == "float32"))
        toks = [torch.randint(0, c["vocab"], (n,), generator=torch.Generator().manual_seed(n)).tolist() for n in (LONG, 61, 97, 2)]
        wd = {k: v.double() for k, v in w.items()}
        _cache[key] = (c, d, toks, [O.forward(c, wd, t).float() for t in toks], [x.float() for x in O.forward(c, wd, toks[1], True)[1]])
    c, d, toks, ref, _ = _cache[key]
    if (name, dtype) not in _cache:
        cfg, ck = open_checkpoint(str(d))
        _cache[name, dtype] = BlockModel.from_state_dict(cfg, ck, DEV, page=16, dtype=dtype)
    return c, _cache[name, dtype], toks, ref


def engine(m, **kw):
    kw = {"max_seqs": 4, "max_ctx": 256, "prefill_chunk": 64, "max_batch": 4} | kw
    return Engine(m, **kw)


TOL = {"float32": 2e-4, "bfloat16": 6e-2}
rms = lambda a, b: float(((a - b) - (a - b).mean(-1, keepdim=True)).pow(2).mean(-1).sqrt().max() / b.std(-1).mean())


def feed(eng, sid, toks, cuts, decode_from=None):
    """All logits of one sequence fed in portions of the given sizes (cycled)."""
    out, p, k = [], 0, 0
    while p < len(toks):
        n = 1 if decode_from is not None and p >= decode_from else min(cuts[k % len(cuts)], len(toks) - p)
        out.append(eng.step([Portion(sid, toks[p: p + n], list(range(n)))], return_logits=True)[0][1])
        p, k = p + n, k + 1
    return torch.cat(out)


@pytest.mark.parametrize("name", list(O.MODELS))
def test_residual_stream_after_every_layer_run(tmp_path_factory, name):
    c, m, toks, _ = load(tmp_path_factory, name, "float32")
    eng = engine(m)
    m.drift = {}
    s = eng.create_sequence()
    eng.step([Portion(s, toks[1], [])])
    got, m.drift = m.drift, None
    eng.free_sequence(s)
    want = _cache[name, "float32", "files"][4]
    assert len(got) == len(want)
    for i, x in enumerate(want):
        assert err(got[f"layer{i:03d}.resid"], x) < 1e-4, i


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(O.MODELS))
def test_prompts_portions_and_decoding_match_the_oracle(tmp_path_factory, name, dtype):
    if (name, dtype) == ("ones", "bfloat16"):
        pytest.skip("a norm over one channel is a sign, which rounding turns")
    c, m, toks, ref = load(tmp_path_factory, name, dtype)
    eng = engine(m)
    for cuts, dec in (([LONG], None), ([2], None), ([3, 64, 2, 65], 150), ([17], None), ([1], None), ([100, 2, 9], 110)):
        sid = eng.create_sequence()
        e = rms(feed(eng, sid, toks[0], cuts, dec), ref[0])
        assert e < TOL[dtype], (cuts, dec, e)
        assert eng.seq_len(sid) == LONG
        eng.free_sequence(sid)


@pytest.mark.parametrize("name", ["tiles", "odd", "wide"])
def test_long_prompt_runs_beside_other_requests(tmp_path_factory, name):
    """Runs long enough for keys and values written out per head, the second one starting behind the window's first key."""
    c, m, toks, ref = load(tmp_path_factory, name, "bfloat16")
    eng = engine(m, prefill_chunk=256)
    a, b, d = (eng.create_sequence() for _ in range(3))
    eng.step([Portion(b, toks[1][:4], [])])
    res = eng.step([Portion(d, toks[2][:3], [0, 2]), Portion(a, toks[0][:140], list(range(140))), Portion(b, toks[1][4:5], [0])], return_logits=True)
    assert rms(res[0][1], ref[2][[0, 2]]) < 6e-2 and rms(res[1][1], ref[0][:140]) < 6e-2 and rms(res[2][1], ref[1][4:5]) < 6e-2
    e = engine(m, prefill_chunk=256)
    s = e.create_sequence()
    assert rms(feed(e, s, toks[0], [60, 140]), ref[0]) < 6e-2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["odd", "tiles"])
def test_mixed_batches_with_reused_pages_and_slots(tmp_path_factory, name, dtype):
    """Unequal requests in one batch against each alone, in a pool that only holds what is live: pages and slots go round several times;
    requests pause, portions sit beside single tokens, a request of two tokens comes and goes."""
    c, m, toks, ref = load(tmp_path_factory, name, dtype)
    pages = (LONG + 15) // 16 + (61 + 15) // 16 + (97 + 15) // 16 + 1
    eng = engine(m, num_pages=pages)
    g = torch.Generator().manual_seed(4)
    live, at, worst, done = {}, {}, 0.0, 0
    sizes = [1, 1, 2, 30, 1, 64, 3, 1, 90]
    for step in range(700):
        for r in range(4):
            if r not in live and (r != 3 or step % 7 == 0):
                live[r], at[r] = eng.create_sequence(), 0
        go = [r for r in live if torch.rand(1, generator=g) < 0.8] or list(live)
        parts = {r: min(sizes[int(torch.randint(0, len(sizes), (1,), generator=g))], len(toks[r]) - at[r]) for r in go}
        res = eng.step([Portion(live[r], toks[r][at[r]: at[r] + n], [0, n - 1] if n > 1 else [0]) for r, n in parts.items()], return_logits=True)
        for (r, n), (nx, lg) in zip(parts.items(), res):
            rows = [at[r], at[r] + n - 1] if n > 1 else [at[r]]
            worst = max(worst, rms(lg, ref[r][rows]))
            assert nx == lg.argmax(-1).tolist()
            at[r] += n
            if at[r] == len(toks[r]):
                eng.free_sequence(live.pop(r))
                done += 1
        assert worst < TOL[dtype], (step, parts, worst)
        if done >= 24:
            break
    for r in list(live):
        eng.free_sequence(live.pop(r))
    assert done >= 24 and eng.free_page_count() == pages


@pytest.mark.parametrize("name,dtype", [("tiles", "bfloat16"), ("wide", "bfloat16"), ("odd", "float32")])
def test_long_decoding_through_the_captured_step(tmp_path_factory, name, dtype):
    """Three sequences decode together until every window has passed over decoded tokens."""
    c, m, toks, ref = load(tmp_path_factory, name, dtype)
    eng = engine(m)
    sids = [eng.create_sequence() for _ in range(3)]
    starts = [5, 1, 40]
    for s, t, n in zip(sids, toks, starts):
        eng.prefill(s, t[:n])
    for k in range(57):
        on = [j for j in range(3) if starts[j] + k < len(toks[j])]
        _, lg = eng.decode([sids[j] for j in on], [toks[j][starts[j] + k] for j in on], return_logits=True)
        for row, j in zip(lg, on):
            assert rms(row[None], ref[j][starts[j] + k][None]) < TOL[dtype], (j, k)
    for p in range(starts[0] + 57, LONG):
        _, lg = eng.decode([sids[0]], [toks[0][p]], return_logits=True)
        assert rms(lg, ref[0][p: p + 1]) < TOL[dtype], p


def test_a_wide_decode_batch_and_a_step_larger_than_a_pass(tmp_path_factory):
    """Twelve sequences of unequal length decode in one step (the many-row forms of every kernel over single tokens)."""
    c, m, toks, ref = load(tmp_path_factory, "tiles", "bfloat16")
    eng = engine(m, max_seqs=12, max_batch=12)
    sids, at = [eng.create_sequence() for _ in range(12)], [3 + 15 * j for j in range(12)]
    for s, a in zip(sids, at):
        eng.prefill(s, toks[0][:a])
    for k in range(18):
        _, lg = eng.decode(sids, [toks[0][a + k] for a in at], return_logits=True)
        assert rms(lg, ref[0][[a + k for a in at]]) < TOL["bfloat16"], k
    c, m, toks, ref = load(tmp_path_factory, "odd", "float32")
    eng = engine(m, prefill_chunk=32)
    a, b, d = (eng.create_sequence() for _ in range(3))
    eng.step([Portion(b, toks[1][:1], [])])
    res = eng.step([Portion(a, toks[0], [0, 70, LONG - 1]), Portion(b, toks[1][1:2], [0]), Portion(d, toks[2], list(range(97)))], return_logits=True)
    assert rms(res[0][1], ref[0][[0, 70, LONG - 1]]) < 2e-4 and rms(res[1][1], ref[1][1:2]) < 2e-4 and rms(res[2][1], ref[2]) < 2e-4


def test_forks_anchored_rewinds_and_hibernation_keep_cache_and_state(tmp_path_factory):
    c, m, toks, ref = load(tmp_path_factory, "odd", "float32")
    eng = engine(m)
    eng.enable_kv_tiering(32)
    a = eng.create_sequence()
    eng.prefill(a, toks[0][:70])
    b = eng.fork_sequence(a)
    eng.anchor(a)
    eng.forward_rows(a, toks[0][70:76])
    eng.rewind(a, 73)
    eng.hibernate(b)
    assert rms(eng.step([Portion(a, toks[0][73:90], [16])], return_logits=True)[0][1], ref[0][89:90]) < 2e-4
    assert rms(eng.step([Portion(b, toks[0][70:72], [1])], return_logits=True)[0][1], ref[0][71:72]) < 2e-4
    assert rms(eng.forward_rows(b, toks[0][72:75]), ref[0][72:75]) < 2e-4
    with pytest.raises(RuntimeError):
        eng.fork_sequence(a, 20)                                            # the state only exists at the frontier


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_server_scheduler(tmp_path_factory, dtype):
    """Requests that join, decode together and leave get the tokens of ``Engine.generate`` alone; in fp32 these are the oracle's."""
    from layerstorm_b200.serving.orchestrator import InferenceRequest, Orchestrator, SamplingParams
    c, m, toks, _ = load(tmp_path_factory, "odd", dtype)
    eng = engine(m, max_seqs=8)
    prompts, gens = [toks[0][:90], toks[1], toks[2][:40], toks[0][100:103], toks[2]], [9, 14, 5, 11, 7]
    orch = Orchestrator(eng, eos_token_ids=[], max_batch=4, prefill_slice_tokens=16)
    reqs = [InferenceRequest(f"g{j}", list(p), SamplingParams(max_tokens=n, ignore_eos=True)) for j, (p, n) in enumerate(zip(prompts, gens))]
    for r in reqs:
        orch.submit_request(r)
    for _ in range(300):
        if not orch.step():
            break
    assert all(r.done.is_set() and r.error is None for r in reqs), [r.error for r in reqs]
    assert orch.mixed_steps > 3
    orch.prefix.clear()
    assert not eng.seqs
    if dtype == "float32":
        w = {k: v.to(B16).float() for k, v in O.random_model(c, 11).items()}
        for p, n, r in zip(prompts, gens, reqs):
            lg = O.forward(c, w, list(p) + list(r.output_ids))[len(p) - 1: -1]
            best = lg.max(-1).values
            assert len(r.output_ids) == n and all(float(best[j] - lg[j, t]) < 1e-3 for j, t in enumerate(r.output_ids))
            assert eng.generate(p, n) == list(r.output_ids)
    else:
        alone = [eng.generate(p, n) for p, n in zip(prompts, gens)]
        assert sum(a == list(r.output_ids) for a, r in zip(alone, reqs)) >= 3        # ties of rounded activations may fall either way


def test_random_layers_run_and_sample():
    from layerstorm_b200.models.config import get_preset
    m = BlockModel.random_init(get_preset("tiny-nivasun"), DEV, seed=1)
    eng = engine(m)
    assert len(eng.generate(list(range(2, 40)), 6)) == 6 and eng.kernel_launches > 0
    s = eng.create_sequence()
    eng.prefill(s, list(range(20)))
    assert 0 <= eng.decode([s], [3], sample=(0.8, 5, 0.9, 7))[0] < 320
    m.set_layer_skip([1, 2])
    assert not m.skip_layers                                                 # layers of the loop always run
    m.set_layer_skip([])


def test_trace_replay_and_the_server_boot_a_checkpoint_directory(tmp_path_factory, tmp_path):
    import json

    import numpy as np

    from layerstorm_b200.cli import serve, trace_run
    c, m, toks, ref = load(tmp_path_factory, "odd", "bfloat16")
    d = _cache["odd", "bfloat16", "files"][1]
    args = serve.build_parser().parse_args(["--model", str(d), "--max-sequence-length", "512", "--max-concurrent", "3", "--tokenizer-mode", "byte"])
    cfg, shape, ckpt, _ = serve.resolve_config(args)
    eng = serve.build_engine(cfg, shape, ckpt, args)
    assert isinstance(eng.model, BlockModel) and eng.supports_mixed_steps and eng.model.kv_fmt == "bf16"
    s = eng.create_sequence()
    _, lg = eng.prefill(s, toks[1], want_logits=True)
    assert rms(lg[None], ref[1][-1:]) < TOL["bfloat16"]
    said = []
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[1][:30], "want": [4]}, {"id": "b", "tokens": toks[2][:2]}]},
             {"step": 1, "entries": [{"id": "b", "tokens": toks[2][2:3], "want": [0]}, {"id": "a", "tokens": toks[1][30:], "want": [0, 30]}], "end": ["a", "b"]}]
    trace_run.replay(engine(m), [json.dumps(x) for x in steps], str(tmp_path), said.append)
    assert said == ["done 0", "done 1"]
    got = [torch.from_numpy(np.fromfile(tmp_path / f"{k}.f32", dtype="<f4")).view(-1, c["vocab"]) for k in (0, 1)]
    assert rms(got[0], ref[1][4:5]) < TOL["bfloat16"] and rms(got[1], torch.stack([ref[2][2], ref[1][30], ref[1][60]])) < TOL["bfloat16"]
