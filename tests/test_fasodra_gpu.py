"""Fasodra on the device against the plain evaluation in fasodra_oracle.py: every mechanism alone, then whole models of several geometries through
the engine - prompts, decoding, portions, mixed batches, reused pages and slots, generation through the server's scheduler."""
import pytest
import torch

pytestmark = pytest.mark.gpu

import fasodra_oracle as O
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


# ------------------------------------------------------------------------------------------------ attention
class Paged:
    """Sequences laid out over shuffled cache pages; rows of a step = runs of tokens of some of them."""

    def __init__(self, H, G, dk, dv, page, lens, f32, seed=0):
        self.H, self.G, self.dk, self.dv, self.page, self.f32 = H, G, dk, dv, page, f32
        self.dkp, self.dvp = nat.call("lsb_attn_head_pad", dk), nat.call("lsb_attn_head_pad", dv)
        g = torch.Generator().manual_seed(seed)
        self.max_pages = max((n + page - 1) // page for n in lens)
        n_pages = len(lens) * self.max_pages + 3
        self.bt = torch.randperm(n_pages, generator=g)[: len(lens) * self.max_pages].view(len(lens), -1).int().to(DEV)
        self.dt = F32 if f32 else B16
        self.cache = torch.full((n_pages, page, G * (self.dkp + self.dvp)), 7.5, dtype=self.dt, device=DEV)     # stale values everywhere

    def run(self, parts, norm=0, bias=(None, None, None), wq=None, wk=None, rot=0, base=1e4, eps=1e-5, scale=1.0, chunk=0, rel=None, gate=False, out_scale=1.0, NS=1):
        """parts: (sequence, first position, q [n, H dk], k [n, G dk], v [n, G dv], gate logits [n, H]); rel: [H, distances]."""
        H, G, dk, dv = self.H, self.G, self.dk, self.dv
        proj = torch.cat([torch.cat(p[2:], 1) for p in parts]).float().to(DEV).contiguous()
        R, n = proj.shape[0], [len(p[2]) for p in parts]
        seq, pos = i32([s for s, p0, q, *_ in parts for _ in range(len(q))]), i32([p0 + j for s, p0, q, *_ in parts for j in range(len(q))])
        q = torch.zeros(R, H, self.dkp, dtype=self.dt, device=DEV)
        out = torch.full((R, H * dv + 8), 3.0, dtype=self.dt, device=DEV)
        op, ml = torch.zeros(R * H * NS * self.dvp, device=DEV), torch.zeros(R * H * NS * 2, device=DEV)
        inv = torch.tensor([base ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float64, device=DEV) if rot else None
        oq, ok, ov, og = 0, H * dk, (H + G) * dk, (H + G) * dk + G * dv
        nat.call("lsb_attn_head_prep", proj, proj.shape[1], oq, ok, ov, *(dev(b) for b in bias), norm, dev(wq), dev(wk), eps, rot, 0, inv, None, 1, q, self.cache, self.bt,
                 self.max_pages, seq, pos, R, H, G, dk, dv, self.dkp, self.dvp, self.page, int(self.f32))
        rel = dev(rel)
        nat.call("lsb_attn", q, self.cache, self.bt, self.max_pages, self.page, seq, pos, i32([sum(n[:j]) for j in range(len(n))]), i32(n), len(n), max(n), proj,
                 proj.shape[1], og if gate else -1, out, H * dv + 8, op, ml, NS, R, H, G, dk, dv, self.dkp, self.dvp, 0, scale, None, 1, chunk, rel,
                 rel.shape[1] if rel is not None else 0, out_scale, None, 1, int(self.f32))
        torch.cuda.synchronize()
        assert float((out[:, H * dv:].float() - 3.0).abs().max()) == 0
        return out[:, : H * dv].float().cpu()


GEOMETRIES = [(4, 2, 32, 32), (6, 1, 24, 40), (8, 8, 64, 64), (3, 3, 128, 96), (20, 1, 64, 128), (2, 1, 200, 256), (2, 2, 20, 272), (33, 1, 40, 24)]


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,G,dk,dv", GEOMETRIES)
def test_chunked_attention_sees_exactly_its_chunk(H, G, dk, dv, f32):
    """One key stands out for every query: the token itself, the first of its chunk, the last of the chunk before (then a nearer decoy must win), one at a
    page border.  Prompt runs of unequal length cut inside chunks, then single rows with and without key splits.  The learned bias turns scores round at
    single distances, so that a table read one entry off shows."""
    if f32 and (H, G) not in ((6, 1), (3, 3)):
        pytest.skip("the CUDA-core kernel has one form")
    T, C, page, reach = 150, 37, 16, 60
    g = torch.Generator().manual_seed(H * 100 + dk)
    lens, data = [T, T - 29], []
    for n in lens:
        k = torch.nn.functional.normalize(torch.randn(n, G, dk, generator=g), dim=-1) * dk ** 0.5
        v, q = torch.randn(n, G, dv, generator=g), torch.empty(n, H, dk)
        for i in range(n):
            for h in range(H):
                at = (i, i // C * C, i // C * C - 1, max(i // page * page, i // C * C), max(i // page * page - 1, i // C * C), i - 1)[(i + h) % 6]
                q[i, h] = 40.0 / dk * k[max(0, at), h // (H // G)] + (12.0 / dk * k[i, h // (H // G)] if at < i // C * C else 0.0)
        data.append((exactly(q.reshape(n, -1), f32), exactly(k.reshape(n, -1), f32), exactly(v.reshape(n, -1), f32), torch.randn(n, H, generator=g)))
    table = 6.0 * torch.randn(reach, H, generator=g)                      # one row per distance
    rel = table[torch.arange(T).clamp(max=reach - 1)]
    for chunk, bias in ((C, True), (C, False), (0, True)):
        b = None
        if bias:
            b = rel[(torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)].permute(2, 0, 1)
        ref = [O.attention(q.view(-1, H, dk), k.view(-1, G, dk), v.view(-1, G, dv), 0.9, None if b is None else b[:, : len(q), : len(q)], chunk)
               .mul(0.7 * torch.sigmoid(gt)[..., None]).flatten(1) for q, k, v, gt in data]
        kw = dict(chunk=chunk, scale=0.9, rel=table.T if bias else None, gate=True, out_scale=0.7)
        tol = 2e-5 if f32 else 8e-3
        P = Paged(H, G, dk, dv, page, lens, f32)
        cut = lambda s, a, z: (s, a, *(t[a:z] for t in data[s]))
        out = P.run([cut(0, 0, T), cut(1, 0, 3)], **kw)
        assert err(out, torch.cat([ref[0], ref[1][:3]])) < tol
        assert err(P.run([cut(1, 3, 70)], **kw), ref[1][3:70]) < tol
        for a in range(70, lens[1]):                                     # decoded
            for NS in ((1, 3) if a % 10 == 0 or a % C < 2 else (1,)):
                assert err(P.run([cut(1, a, a + 1)], NS=NS, **kw), ref[1][a: a + 1]) < tol, (a, NS)
        P = Paged(H, G, dk, dv, page, lens, f32, seed=9)
        outs = [P.run([cut(0, a, a + 2), cut(1, a, a + 2)], NS=1 + a // 2 % 2, **kw) for a in range(0, 120, 2)]
        assert err(torch.cat([o[:2] for o in outs]), ref[0][:120]) < tol and err(torch.cat([o[2:] for o in outs]), ref[1][:120]) < tol
        P = Paged(H, G, dk, dv, page, lens, f32, seed=5)
        outs = [P.run([cut(0, a, min(T, a + 19))], **kw) for a in range(0, T, 19)]
        assert err(torch.cat(outs), ref[0]) < tol


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("norm", [0, 1, 2])
@pytest.mark.parametrize("dk,dv,rot", [(24, 40, 6), (64, 32, 64), (96, 96, 32), (18, 8, 2)])
def test_biases_head_norms_and_rotation(norm, dk, dv, rot, f32):
    """Against the oracle's steps in fp32: bias in front of the norm, norm in front of the rotation, values neither; far positions keep their angles."""
    H, G, n, eps = 6, 2, 40, 1e-2
    g = torch.Generator().manual_seed(dk)
    q, k, v = (torch.randn(n, w, generator=g) * 2 for w in (H * dk, G * dk, G * dv))
    b = [torch.randn(w, generator=g) for w in (H * dk, G * dk, G * dv)]
    wq, wk = 1 + 0.3 * torch.randn(dk, generator=g), 1 + 0.3 * torch.randn(dk, generator=g)
    x, y = (q + b[0]).view(n, H, dk), (k + b[1]).view(n, G, dk)
    if norm:
        x, y = O.rms(x, eps), O.rms(y, eps)
    if norm == 2:
        x, y = x * wq, y * wk
    x, y = O.rotate_half(x.double(), rot, 300.0).float(), O.rotate_half(y.double(), rot, 300.0).float()
    scale = 0.3 if norm else 0.05                                          # raw heads are five times as large
    ref = O.attention(x, y, (v + b[2]).view(n, G, dv), scale).flatten(1)
    kw = dict(norm=norm, bias=b, wq=wq, wk=wk, rot=rot, base=300.0, eps=eps, scale=scale)
    gt = torch.zeros(n, H)
    P = Paged(H, G, dk, dv, 16, [n], f32)
    assert err(P.run([(0, 0, q, k, v, gt)], **kw), ref) < (3e-5 if f32 else 1.5e-2)
    P = Paged(H, G, dk, dv, 16, [n], f32, seed=1)
    outs = [P.run([(0, a, q[a: a + 1], k[a: a + 1], v[a: a + 1], gt[:1])], **kw) for a in range(n)]
    assert err(torch.cat(outs), ref) < (3e-5 if f32 else 1.5e-2)


def test_rotation_at_far_positions():
    """Two tokens at far positions of an otherwise empty table: their score depends on the distance alone."""
    H, dk, rot, far = 1, 8, 8, 70000
    q, k, v = torch.randn(2, dk), torch.randn(2, dk), torch.eye(2, dk)
    outs = []
    for p0 in (0, far):
        P = Paged(H, 1, dk, dk, 16, [p0 + 2], True)
        P.cache.zero_()
        outs.append(P.run([(0, p0, q, k, v, torch.zeros(2, 1))], rot=rot, base=10.0, chunk=far)[1])        # the chunk starts at the first of the two
    assert err(outs[1], outs[0]) < 1e-4


# ------------------------------------------------------------------------------------------------ delta rule with a decay per head
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,G,dk,dv,taps", [(4, 2, 32, 64, 4), (6, 3, 24, 20, 3), (2, 1, 48, 96, 1), (2, 2, 128, 128, 4), (1, 1, 160, 72, 2), (3, 3, 1, 1, 2)])
def test_delta_rule_with_head_decays_and_full_gates(H, G, dk, dv, taps, f32):
    """Token by token, chunk-parallel and as one kernel, in portions of every short length, on interleaved state slots."""
    T, eps = 170, 1e-5
    g = torch.Generator().manual_seed(dk)
    n = lambda *s: torch.randn(*s, generator=g)
    conv = [torch.rand(c, taps, generator=g) * 2 - 1 for c in (G * dk, G * dk, H * dv)]
    a_log, dt, onorm = torch.rand(H, generator=g) * 4 - 3.5, torch.rand(H, generator=g) * 3 - 3, 1 + 0.2 * n(dv)
    widths = [G * dk, G * dk, H * dv, H, H, H * dv]
    offs = [sum((x + 7) // 8 * 8 for x in widths[:j]) for j in range(6)]
    ld = offs[-1] + (widths[-1] + 7) // 8 * 8
    xs = [[n(T, w) for w in widths] for _ in range(2)]

    def reference(x):
        q, k, v = (O.short_conv(x[j].double(), conv[j].double()) for j in range(3))
        q, k = (O.unit(t.view(T, G, dk)).repeat_interleave(H // G, 1) for t in (q, k))
        dec = torch.exp(-torch.exp(a_log.double()) * O.softplus(x[4].double() + dt))
        o, S = O.delta_rule(q * dk ** -0.5, k, v.view(T, H, dv), dec, torch.sigmoid(x[3].double()))
        return ((O.rms(o, eps) * onorm).flatten(1) * O.silu(x[5].double())).float(), S.float()

    refs = [reference(x) for x in xs]
    tol = 3e-5 if f32 else 1e-2
    for form in ["rows"] + (["chunk"] if dk <= 128 else []) + (["few"] if dv <= nat.call("lsb_delta_few_max_dv", dk) else []):
        state, hist = torch.zeros(3, H, dv, nat.call("lsb_delta_key_pad", dk), device=DEV), torch.zeros(3, H, 2 * dk + dv, taps - 1, device=DEV)
        at = [0, 0]
        for cuts in [(1, 2), (2, 1), (40, 70), (7, 1), (64, 3), (1, 93), (55, 0)] if form != "few" else [(1, 1), (2, 3), (8, 1)] * 14:
            parts = [(s, j, c) for s, j, c in ((2, 0, cuts[0]), (0, 1, cuts[1])) if c]
            m = [c for _, _, c in parts]
            R = sum(m)
            proj, r0 = torch.zeros(R, ld, device=DEV), 0
            for _, j, c in parts:
                for o, t in zip(offs, xs[j]):
                    proj[r0: r0 + c, o: o + t.shape[1]] = t[at[j]: at[j] + c].to(DEV)
                r0 += c
            out = torch.zeros(R, H * dv + 4, dtype=F32 if f32 else B16, device=DEV)
            longs = [c for c in m if c >= 16] if form == "chunk" else []
            chunks = sum((c + 63) // 64 for c in longs)
            scratch = torch.full((nat.call("lsb_delta_scratch_floats", R, H, dk, dv, 0, 0),), float("nan"), device=DEV)
            cw = torch.full((max(1, nat.call("lsb_delta_chunk_floats", chunks, H, dk)),), float("nan"), device=DEV)
            e = torch.zeros(1, dtype=I32, device=DEV)
            nat.call("lsb_delta_forward", proj, ld, *offs, 0, 0, None, None, None, None, *(c.to(DEV) for c in conv), dev(torch.exp(a_log)), dev(dt), dev(onorm), state, hist,
                     i32([sum(m[:j]) for j in range(len(m))]), i32(m), i32([s for s, _, _ in parts]), out, H * dv + 4, len(m), R, H, G, dk, dv, taps, 0, dk ** -0.5, 0.0,
                     eps, int(f32), int(form == "few"), scratch, len(m) - len(longs), len(longs), chunks, 16, cw, e)
            torch.cuda.synchronize()
            r0 = 0
            for _, j, c in parts:
                assert err(out[r0: r0 + c, : H * dv], refs[j][0][at[j]: at[j] + c]) < tol, (form, at, cuts)
                r0, at[j] = r0 + c, at[j] + c
        if at[0] == T:
            assert err(state[2, ..., :dk].transpose(1, 2), refs[0][1]) < 3e-5
        assert float(state[1].abs().max()) == 0


# ------------------------------------------------------------------------------------------------ time mixing
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("width", [12, 136, 2048])
def test_token_shift_takes_the_predecessor_across_steps(width, f32):
    """The predecessor of a run's first row is the kept input of its own slot, zeros for a fresh one; every other row's is the row in front of it."""
    g = torch.Generator().manual_seed(width)
    n = [3, 1, 5]
    R, x = sum(n), exactly(torch.randn(sum(n), width, generator=g), f32)
    mu, prev = torch.rand(5, width, generator=g), torch.randn(4, width, generator=g)
    prev[2] = 0
    xs = torch.zeros(5, R + 3, width, dtype=F32 if f32 else B16, device=DEV)
    nat.call("lsb_tmix_shift", x.to(xs.dtype).to(DEV), width, dev(prev), dev(mu), xs, xs.stride(0), i32([0, 3, 4]), i32(n), i32([1, 3, 2]), 3, R, int(f32))
    before = torch.cat([prev[1:2], x[0:2], prev[3:4], prev[2:3], x[4:8]])
    want = torch.stack([x + (before - x) * mu[s] for s in range(5)])
    assert err(xs[:, :R], want) < (1e-6 if f32 else 5e-3) and float(xs[:, R:].abs().sum()) == 0


class Mix:
    def __init__(self, H, dk, dv, rank=12, f32=True, seed=0, slots=3):
        g = torch.Generator().manual_seed(seed)
        n = lambda *s: torch.randn(*s, generator=g)
        self.s, self.f32, self.rank = (H, dk, dv), f32, (rank + 7) // 8 * 8
        self.w2, self.w0 = exactly(n(H * dk, rank) * 1.5 / rank ** 0.5, f32), torch.rand(H * dk, generator=g) * 6 - 5
        self.u, self.onorm = n(H, dk), 1 + 0.2 * n(H * dv)
        self.widths = [H * dk, H * dk, H * dv, H * dv, rank]               # r, k, v, g, w
        self.offs = [sum((x + 7) // 8 * 8 for x in self.widths[:j]) for j in range(5)]
        self.ld = self.offs[-1] + self.rank
        w2 = torch.nn.functional.pad(self.w2, (0, self.rank - rank)).to(F32 if f32 else B16).to(DEV).contiguous()
        self.dw2, self.dw22 = w2, torch.cat([w2, w2], 1).contiguous()
        self.state = torch.zeros(slots, H, dv, nat.call("lsb_tmix_key_pad", dk), device=DEV)
        self.prev = torch.zeros(slots, 16, device=DEV)

    def inputs(self, T, seed):
        g = torch.Generator().manual_seed(seed)
        return [torch.randn(T, w, generator=g) for w in self.widths]

    def reference(self, x, eps=1e-5):
        H, dk, dv = self.s
        r, k, v = (t.double().view(len(t), H, -1) for t in x[:3])
        w = torch.exp(-torch.exp(torch.tanh(x[4].double()) @ self.w2.double().T + self.w0)).view(len(r), H, dk)
        o, S = O.time_mixing(r, k, v, w, self.u.double())
        return (O.rms(o, eps).flatten(1) * self.onorm * O.silu(x[3].double())).float(), S.float()

    def run(self, parts, form, eps=1e-5):
        """parts: (slot, inputs); form: few | chunk."""
        H, dk, dv = self.s
        n = [len(p[1][0]) for p in parts]
        R, r0 = sum(n), 0
        proj = torch.zeros(R, self.ld, device=DEV)
        for (_, x), m in zip(parts, n):
            for o, t in zip(self.offs, x):
                proj[r0: r0 + m, o: o + t.shape[1]] = t.to(DEV)
            r0 += m
        dt = F32 if self.f32 else B16
        x = torch.arange(R * 16, device=DEV).view(R, 16).to(dt).contiguous()
        out, e = torch.zeros(R, H * dv + 4, dtype=dt, device=DEV), torch.zeros(1, dtype=I32, device=DEV)
        chunks = sum((m + 63) // 64 for m in n)
        scratch = torch.full((nat.call("lsb_tmix_scratch_floats", R, chunks, H, dk, dv, self.rank),), float("nan"), device=DEV)
        nat.call("lsb_tmix_forward", proj, self.ld, *self.offs, self.rank, self.dw2, None if self.f32 else self.dw22, dev(self.w0), dev(self.u), dev(self.onorm),
                 self.state, self.prev, x, 16, i32([sum(n[:j]) for j in range(len(n))]), i32(n), i32([p[0] for p in parts]), out, H * dv + 4, len(n), R, H, dk, dv,
                 eps, int(self.f32), int(form == "few"), scratch, chunks, e)
        torch.cuda.synchronize()
        assert int(e[0]) == 0 and float(out[:, H * dv:].abs().sum()) == 0
        for (s, _), last in zip(parts, torch.tensor(n).cumsum(0).tolist()):
            assert torch.equal(self.prev[s], x[last - 1].float())           # the kept input: the run's last row
        return out[:, : H * dv].float().cpu()


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,dk,dv", [(4, 32, 32), (3, 24, 20), (2, 64, 64), (5, 12, 40), (2, 128, 128), (1, 100, 130), (2, 160, 160), (1, 1, 1), (2, 48, 300)])
def test_time_mixing_forms_agree_with_the_recurrence(H, dk, dv, f32):
    T, tol = 170, 4e-5 if f32 else 1e-2
    for form in ["few"] + (["chunk"] if dk <= 128 else []):
        M = Mix(H, dk, dv, f32=f32, seed=dk)
        a, b = M.inputs(T, 1), M.inputs(T, 2)
        (ra, Sa), (rb, _) = M.reference(a), M.reference(b)
        sl = lambda x, i, j: [t[i:j] for t in x]
        i = j = 0
        for na, nb in [(1, 2), (2, 1), (40, 70), (7, 1), (64, 3), (1, 93), (55, 0)] if form == "chunk" else [(1, 1), (2, 3), (8, 1), (13, 2), (40, 30), (1, 0), (105, 9)]:
            out = M.run([(2, sl(a, i, i + na))] + ([(0, sl(b, j, j + nb))] if nb else []), form)
            assert err(out[:na], ra[i: i + na]) < tol, (form, i, na)
            assert nb == 0 or err(out[na:], rb[j: j + nb]) < tol, (form, j, nb)
            i, j = i + na, j + nb
        assert i == T and err(M.state[2, ..., :dk].transpose(1, 2), Sa) < 4e-5
        assert float(M.state[1].abs().max()) == 0 and float(M.state[..., dk:].abs().sum()) == 0


def test_time_mixing_survives_strong_and_weak_decays():
    """Neighbouring tokens and channels with decay factors of exactly 0 and of ~1: nothing overflows, and weak decays keep their digits behind strong ones."""
    M = Mix(2, 32, 32, seed=6)
    M.w2.zero_()
    M.dw2.zero_()
    M.w0 = torch.linspace(-9.0, 7.0, 64)[torch.randperm(64, generator=torch.Generator().manual_seed(1))]
    x = M.inputs(150, 8)
    ref = M.reference(x)[0]
    for s, f in enumerate(("few", "chunk")):
        out = M.run([(s, x)], f)
        assert torch.isfinite(out).all() and err(out, ref) < 4e-5
    M = Mix(1, 32, 32, rank=8, seed=7)                                     # strength alternating from token to token
    M.w2.fill_(3.0)
    M.dw2.fill_(3.0)
    M.w0 = torch.full((32,), -7.0)
    x = M.inputs(150, 9)
    x[4] = torch.where((torch.arange(150) % 7 == 3)[:, None], 1.0, -1.0).expand(150, 8).contiguous()
    ref = M.reference(x)[0]
    for s, f in enumerate(("few", "chunk")):
        assert err(M.run([(s, x)], f), ref) < 4e-5


@pytest.mark.parametrize("M,N,K", [(1, 5, 136), (3, 40, 384), (7, 129, 4096), (4, 16, 8)])
def test_products_with_an_input_per_run_of_weight_rows(M, N, K):
    g = torch.Generator().manual_seed(N)
    rows = [0]
    for _ in range(4):
        rows.append(rows[-1] + (N + 7) // 8 * 8)
    tot, x = rows[-1] + 24, torch.randn(5, M + 2, K, generator=g).to(B16)
    w = torch.randn(tot, K, generator=g).to(B16)
    out = torch.zeros(M, tot + 8, device=DEV)
    nat.call("lsb_gemv_bf16_segs", out, x.to(DEV), w.to(DEV), M, tot, K, K, K, tot + 8, torch.tensor(rows, dtype=I32), 5, x.stride(0))
    want = torch.cat([x[s, :M].float() @ w[a:z].float().T for s, (a, z) in enumerate(zip(rows, rows[1:] + [tot]))], 1)
    assert err(out[:, :tot], want) < 1e-5 and nat.call("lsb_gemv_error") == 0


# ------------------------------------------------------------------------------------------------ streams, experts
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("dim", [37, 136, 1024])
@pytest.mark.parametrize("n", [1, 2, 3, 4, 5, 8])
def test_streams_start_mix_and_end(n, dim, f32):
    R, eps, ld, mult = 5, 1e-2, (dim + 7) // 8 * 8, 0.6
    g = torch.Generator().manual_seed(dim + n)
    r = lambda *s: torch.randn(*s, generator=g)
    pad = lambda t: torch.nn.functional.pad(t, (0, ld - dim)).to(DEV).contiguous()
    w, b, wa, wb = r(dim), r(dim), r(dim), r(dim)
    mix, out, rd = r(n, n), r(n), r(n)
    st, act = torch.full((R, n, ld), 9.0, device=DEV), torch.zeros(R, ld, dtype=F32 if f32 else B16, device=DEV)
    tol = 1e-5 if f32 else 6e-3
    none, no_y = (3, None, None, None), (None, None, None, None, 0, 0, 0)
    e = r(R, dim)
    nat.call("lsb_stream_update", act, ld, st, ld, n, pad(e), None, None, None, ld, None, None, None, None, mult, dev(rd), 1, dev(w), dev(b), None, R, dim, eps, *no_y, int(f32))
    xs = [e] * n
    assert err(act[:, :dim], O.layer_norm(O.read_streams(xs, rd), w, b, eps)) < tol and all(torch.equal(st[:, t, :dim].cpu(), e) for t in range(n))
    # one result, the mean of two normed ones, and an expert sum (one expert not resident)
    E, top = 6, 3
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(R)])
    wt, y = torch.rand(R, top, generator=g), r(R, top, dim)
    slot = torch.arange(E)
    slot[2] = -1
    sub, sub2 = r(R, dim) * 3, r(R, dim) * 0.2
    esum = (torch.where(ids == 2, torch.zeros(()), wt)[..., None] * y).sum(1)
    ye = (pad(y), dev(wt), ids.int().to(DEV), slot.int().to(DEV), top, E, ld)
    for a, b2, ws, yy, res in ((sub, None, (None, None), no_y, sub), (sub, sub2, (dev(wa), dev(wb)), no_y, 0.5 * (O.rms(sub, eps) * wa + O.rms(sub2, eps) * wb)),
                               (None, None, (None, None), ye, esum), (sub, None, (None, None), ye, sub + esum)):
        nat.call("lsb_stream_update", act, ld, st, ld, n, None, None, None if a is None else pad(a), None if b2 is None else pad(b2), ld, *ws, dev(mix), dev(out), mult, dev(rd),
                 1, dev(w), dev(b), None, R, dim, eps, *yy, int(f32))
        xs = O.write_streams(xs, mix, out, mult * res)
        assert all(err(st[:, t, :dim], xs[t]) < 1e-5 for t in range(n))
        assert err(act[:, :dim], O.layer_norm(O.read_streams(xs, rd), w, b, eps)) < tol
    tot = torch.zeros(R, ld, device=DEV)
    nat.call("lsb_stream_update", None, ld, st, ld, n, None, tot, pad(sub), None, ld, None, None, dev(mix), dev(out), mult, None, *none, R, dim, eps, *no_y, int(f32))
    assert err(tot[:, :dim], sum(O.write_streams(xs, mix, out, mult * sub))) < 1e-5


@pytest.mark.parametrize("dtype,R,H,F,E,top", [("float32", 9, 136, 40, 5, 2), ("bfloat16", 5, 136, 40, 5, 3), ("bfloat16", 40, 256, 128, 6, 2), ("bfloat16", 300, 384, 256, 12, 4),
                                               ("bfloat16", 1, 256, 128, 3, 1)])
def test_experts_without_a_gate(dtype, R, H, F, E, top):
    """The weight-streaming and the tensor-core form of the squared-relu experts, and a missing expert's report."""
    from layerstorm_b200.models.device_model import ExpertArena, ModelBase, MoeBuffers, QLinear, expert_layout
    f32 = dtype == "float32"
    dt, fmt = (F32, "f32") if f32 else (B16, "bf16")
    g = torch.Generator().manual_seed(R)
    w = {f"e{j}.{t}": exactly(torch.randn(*s, generator=g) / s[1] ** 0.5, f32) for j in range(E) for t, s in (("up", (F, H)), ("down", (H, F)))}
    x = exactly(torch.randn(R, H, generator=g) * 2, f32)
    arena = ExpertArena(expert_layout(fmt, H, F, gated=False), E, E, torch.device(DEV))
    for j in range(E):
        arena.write_expert(j, None, QLinear(fmt, F, H, w[f"e{j}.up"].to(dt).to(DEV)), QLinear(fmt, H, F, w[f"e{j}.down"].to(dt).to(DEV)))
        arena.slot_of[j] = j
    m, mb = ModelBase(), MoeBuffers()
    m.device = torch.device(DEV)
    z = lambda *s, dtype=F32: torch.zeros(*s, dtype=dtype, device=DEV)
    mb.alloc_moe(z, R, top, E, E, H, F, tc=not f32, act_dtype=dt)
    if mb.tc_ok:
        mb.tc_xs, mb.tc_act = z(R * top, H, dtype=torch.float16), z(R * top, F, dtype=torch.float16)
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(R)])
    mb.ids.copy_(ids.int())
    xd = x.to(dt).to(DEV)
    m.moe_prepare(arena, mb, xd, R, E)
    m.moe_experts(arena, mb, xd, R, E, 0.0, mb.miss, "relu2")
    torch.cuda.synchronize()
    want = torch.stack([torch.cat([O.expert(w, f"e{i}.", x[t: t + 1]) for i in ids[t].tolist()]) for t in range(R)])
    assert err(mb.y.view(R, top, H), want) < (1e-5 if f32 else 1e-2) and int(mb.miss) == 0
    arena.slot_of[int(ids[0, 0])] = -1
    m.moe_experts(arena, mb, xd, R, E, 0.0, mb.miss, "relu2")
    assert int(mb.miss) == int(ids[0, 0]) + 1


def test_softmax_router_divides_by_the_chosen_sum():
    R, E, top = 40, 11, 4
    lg = torch.randn(R, E, generator=torch.Generator().manual_seed(1)) * 3
    ids, wt = O.route(lg, top)
    di, dw = torch.zeros(R, top, dtype=I32, device=DEV), torch.zeros(R, top, device=DEV)
    nat.call("lsb_router_topk_grouped", lg.to(DEV), None, di, dw, R, E, top, 1, 1, 1, 1, 1.0, 0, E, 1)
    assert torch.equal(di.cpu().long(), ids) and err(dw, wt) < 1e-5


# ------------------------------------------------------------------------------------------------ whole models
LONG = 200
_cache = {}


def load(tmp_path_factory, name, dtype):
    """(raw config, device model, tokens, logits of the oracle) of one geometry; models are built once.  The bf16 models have no close routing
    calls: a choice that rounding turns is no error of the kernels (routing itself is checked in fp32)."""
    key = (name, dtype, "files")
    if key not in _cache:
        c = O.MODELS[name]()
        d = tmp_path_factory.mktemp("fasodra")
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
def test_sum_of_the_streams_after_every_layer(tmp_path_factory, name):
    c, m, toks, _ = load(tmp_path_factory, name, "float32")
    eng = engine(m)
    m.drift = {}
    s = eng.create_sequence()
    eng.step([Portion(s, toks[1], [])])
    got, m.drift = m.drift, None
    eng.free_sequence(s)
    for i, x in enumerate(_cache[name, "float32", "files"][4]):
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
    """Three sequences decode together over many chunks of the mask."""
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
    m = BlockModel.random_init(get_preset("tiny-fasodra"), DEV, seed=1)
    eng = engine(m)
    assert len(eng.generate(list(range(2, 40)), 6)) == 6 and eng.kernel_launches > 0
    s = eng.create_sequence()
    eng.prefill(s, list(range(20)))
    assert 0 <= eng.decode([s], [3], sample=(0.8, 5, 0.9, 7))[0] < 320
    m.set_layer_skip([1, 2])
    s = eng.create_sequence()
    assert torch.isfinite(eng.step([Portion(s, [1, 2, 3], [2])], return_logits=True)[0][1]).all()
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
