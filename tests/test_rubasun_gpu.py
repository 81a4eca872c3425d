"""Rubasun on the device against the plain evaluation in rubasun_oracle.py: every mechanism alone, then whole models of several geometries
through the engine - prompts, decoding, portions, mixed batches, reused pages and slots, generation through the server's scheduler."""
import ctypes

import pytest
import torch

pytestmark = pytest.mark.gpu

import rubasun_oracle as O
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


# ------------------------------------------------------------------------------------------------ latent attention
class Paged:
    """Latent rows of sequences laid out over shuffled cache pages; rows of a step = runs of tokens of some of them."""

    def __init__(self, H, dn, dr, dv, dl, page, lens, f32, base=10000.0, seed=0):
        self.sz, self.page, self.f32 = (H, dn, dr, dv, dl), page, f32
        pad = lambda d: nat.call("lsb_latent_pad", d)
        self.dlp, self.drp, self.dnp, self.dt = pad(dl), pad(dr), (dn + 7) // 8 * 8, F32 if f32 else B16
        g = torch.Generator().manual_seed(seed)
        self.max_pages = max((n + page - 1) // page for n in lens)
        n_pages = len(lens) * self.max_pages + 3
        self.bt = torch.randperm(n_pages, generator=g)[: len(lens) * self.max_pages].view(len(lens), -1).int().to(DEV)
        self.cache = torch.full((n_pages, page, self.dlp + self.drp), 7.5, dtype=self.dt, device=DEV)          # stale values everywhere
        self.inv_freq = torch.tensor([base ** (-2 * i / dr) for i in range(dr // 2)], dtype=torch.float64, device=DEV)

    def weights(self, uk, uv, kv_norm):
        H, dn, dr, dv, dl = self.sz
        self.uk = torch.zeros(H, self.dlp, self.dnp, dtype=self.dt, device=DEV)
        self.uk[:, :dl, :dn] = uk.view(H, dn, dl).transpose(1, 2).to(DEV)
        self.uv = torch.zeros(H, dv, self.dlp, dtype=self.dt, device=DEV)
        self.uv[:, :, :dl] = uv.view(H, dv, dl).to(DEV)
        self.kv_norm = kv_norm.to(DEV)
        return self

    def run(self, parts, scale, NS=1, own=True, gate=True, run_rows=None, eps=1e-5):
        """parts: (sequence, first position, q [n, H (dn + dr)], latent projection [n, dl + dr], gate logits [n, H])."""
        H, dn, dr, dv, dl = self.sz
        proj = torch.cat([torch.cat([q, y, gt], 1) for _, _, q, y, gt in parts]).float().to(DEV).contiguous()
        R, D = proj.shape[0], self.dlp + self.drp
        n = [len(p[2]) for p in parts]
        seq, pos = i32([p[0] for p in parts for _ in range(len(p[2]))]), i32([p[1] + j for p in parts for j in range(len(p[2]))])
        row0 = i32([sum(n[:j]) for j in range(len(n))])
        z = lambda *s, dt=self.dt: torch.full(s, float("nan"), dtype=dt, device=DEV)
        ldo = (H * dv + 7) // 8 * 8
        q, qn, ol, out = z(R, H, D), z(R, H, self.dnp, dt=B16), z(R, H, self.dlp), z(R, ldo)
        op, ml = z(R * H * NS * self.dlp, dt=F32), z(R * H * NS * 2, dt=F32)
        e = torch.zeros(1, dtype=I32, device=DEV)
        oq, oy, og = 0, H * (dn + dr), H * (dn + dr) + dl + dr
        nat.call("lsb_latent_query", proj.view(-1)[oq:], proj.shape[1], proj, proj.shape[1], oy if own else -1, self.kv_norm, eps, self.inv_freq, self.uk, q, qn, self.cache, self.bt,
                 self.max_pages, self.page, seq, pos, R, H, dn, self.dnp, dr, dl, int(self.f32), e)
        nat.call("lsb_latent_attn", q, self.cache, self.bt, self.max_pages, self.page, seq, pos, row0, i32(n), len(n), run_rows or max(n), proj, proj.shape[1],
                 og if gate else -1, ol, op, ml, NS, R, H, dl, dr, 0, scale, int(self.f32))
        nat.call("lsb_latent_out", out, ldo, ol, op, ml, nat.call("lsb_latent_partials", NS), self.uv, proj, proj.shape[1], og if gate else -1, 1, seq, R, H, dl, dv, int(self.f32), e)
        torch.cuda.synchronize()
        assert int(e[0]) == 0
        return out[:, : H * dv].float().cpu()


GEOMETRIES = [(4, 32, 16, 32, 64), (6, 24, 10, 20, 40), (16, 128, 64, 128, 512), (33, 40, 32, 16, 128), (70, 8, 2, 9, 17), (1, 1, 2, 1, 1), (20, 64, 64, 96, 256),
              (3, 100, 130, 24, 512), (5, 48, 16, 40, 544)]


def standing_keys(H, dn, dr, dv, dl, lens, f32, base, page, g):
    """Data of sequences in which one key stands out for every (token, head): the token itself, far ones, the rows at page borders; the row right
    behind the token - not to be seen - fits better still.  Returns per sequence (q, latent projection, gate) and (uk, uv, norm)."""
    n = lambda *s: torch.randn(*s, generator=g)
    r = lambda t: exactly(t, f32)
    uk, uv, kvn = r(n(H * dn, dl) / dl ** 0.5), r(n(H * dv, dl) / dl ** 0.5), 1.0 + 0.2 * n(dl)
    data = []
    for T in lens:
        y, gt = n(T, dl + dr), n(T, H)
        pos = torch.arange(T)
        c, kr = O.rms_norm(y[:, :dl], kvn, 1e-5), O.rotate(y[:, dl:], pos, base)
        keys = torch.cat([(c @ uk.T).view(T, H, dn), kr[:, None].expand(T, H, dr)], -1)
        q = torch.empty(T, H, dn + dr)
        for i in range(T):
            for h in range(H):
                back = (0, i, 1, i - i // page * page, i - max(0, i // page * page - 1), i // 2)[(i + h) % 6]
                k, nxt = keys[i - back, h], keys[min(i + 1, T - 1), h]
                q[i, h] = 16.0 * k / k.square().sum() + (22.0 * nxt / nxt.square().sum() if i + 1 < T else 0.0)
        q[..., dn:] = O.rotate(q[..., dn:], -pos, base)                        # the kernel turns it forward again
        data.append((r(q.reshape(T, -1)), y, gt))
    return data, (uk, uv, kvn)


def reference(H, dn, dr, dv, dl, q, y, gt, uk, uv, kvn, scale, base, first=0):
    T = len(q)
    pos = torch.arange(T) + first
    c, kr = O.rms_norm(y[:, :dl], kvn, 1e-5), O.rotate(y[:, dl:], pos, base)
    qq = q.view(T, H, dn + dr)
    qq = torch.cat([qq[..., :dn], O.rotate(qq[..., dn:], pos, base)], -1)
    k = torch.cat([(c @ uk.T).view(T, H, dn), kr[:, None].expand(T, H, dr)], -1)
    o = O.causal_attention(qq.double(), k.double(), (c @ uv.T).view(T, H, dv).double(), scale)
    return (o * torch.sigmoid(gt.double())[..., None]).reshape(T, -1).float()


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,dn,dr,dv,dl", GEOMETRIES)
def test_latent_attention_sees_far_keys_and_nothing_ahead(H, dn, dr, dv, dl, f32):
    """Prompt runs of unequal length in one step, then single rows with and without key splits, then portions of two on other pages."""
    T, page, base, scale = 150, 16, 300.0, 0.9
    lens = [T, T - 29]
    data, (uk, uv, kvn) = standing_keys(H, dn, dr, dv, dl, lens, f32, base, page, torch.Generator().manual_seed(H * 100 + dn))
    ref = [reference(H, dn, dr, dv, dl, *d, uk, uv, kvn, scale, base) for d in data]
    tol = 3e-5 if f32 else (2e-2 if dl > 32 else 6e-2)
    cut = lambda s, a, b: (s, a, *(t[a:b] for t in data[s]))
    tc = not f32 and dl <= 512
    P = Paged(H, dn, dr, dv, dl, page, lens, f32, base).weights(uk, uv, kvn)
    out = P.run([cut(0, 0, T), cut(1, 0, 3)], scale)
    assert err(out, torch.cat([ref[0], ref[1][:3]])) < tol
    assert err(P.run([cut(1, 3, 60)], scale), ref[1][3:60]) < tol
    for a in range(60, lens[1] - 12):                                # decoded
        for NS in ((1, 2, 8, 32) if tc and a % 10 == 0 else (1,)):
            assert err(P.run([cut(1, a, a + 1)], scale, NS), ref[1][a: a + 1]) < tol, (a, NS)
    a = lens[1] - 12
    for NS in ((1, 4, 16) if tc else (1,)):                              # many single rows: the many-row forms of the same step
        rows = [(s, a, *(t[a: a + 1] for t in data[s])) for s in (0, 1)] * 5
        assert err(P.run(rows, scale, NS), torch.cat([ref[0][a: a + 1], ref[1][a: a + 1]] * 5)) < tol
    P = Paged(H, dn, dr, dv, dl, page, lens, f32, base, seed=9).weights(uk, uv, kvn)
    outs = [P.run([cut(0, a, a + 2), cut(1, a, a + 2)], scale, (1, 2, 24)[a // 2 % 3] if tc else 1) for a in range(0, 90, 2)]
    assert err(torch.cat([o[:2] for o in outs]), ref[0][:90]) < tol and err(torch.cat([o[2:] for o in outs]), ref[1][:90]) < tol
    # rows of a layer that reads these rows without appending; without a gate
    out = P.run([(0, 88, *(t[88:90] for t in data[0]))], scale, own=False)
    assert err(out, ref[0][88:90]) < tol
    out = P.run([(0, 88, *(t[88:90] for t in data[0]))], scale, own=False, gate=False)
    gt = torch.sigmoid(data[0][2][88:90])[..., None]
    assert err(out.view(2, H, dv) * gt, ref[0][88:90].view(2, H, dv)) < tol


@pytest.mark.parametrize("H,dn,dr,dv,dl", [g for g in GEOMETRIES if g[1] + g[2] <= 230])
def test_long_runs_over_written_out_keys_and_values(H, dn, dr, dv, dl):
    """The same standing keys through per-head keys and values: a whole prompt, then portions that start inside a page, on rows that were appended
    before and rows of another layer."""
    T, page, base, scale = 150, 16, 300.0, 0.9
    (d,), (uk, uv, kvn) = standing_keys(H, dn, dr, dv, dl, [T], False, base, page, torch.Generator().manual_seed(H * 100 + dn))
    ref = reference(H, dn, dr, dv, dl, *d, uk, uv, kvn, scale, base)
    P = Paged(H, dn, dr, dv, dl, page, [T, T], False, base).weights(uk, uv, kvn)
    up = lambda n: (n + 15) // 16 * 16
    dnw, dvp, drp = up(dn), nat.call("lsb_attn_head_pad", dv), up(dr)
    w = torch.zeros(H * (dnw + dvp), P.dlp, dtype=B16, device=DEV)
    w[: H * dnw].view(H, dnw, P.dlp)[:, :dn, :dl] = uk.view(H, dn, dl).to(DEV)
    w[H * dnw:].view(H, dvp, P.dlp)[:, :dv, :dl] = uv.view(H, dv, dl).to(DEV)
    e, ldo = torch.zeros(1, dtype=I32, device=DEV), (H * dv + 7) // 8 * 8
    for a, b, own in ((0, T, True), (0, 70, True), (70, 73, True), (73, T, True), (20, 101, False)):
        proj = torch.cat([t[a:b] for t in d], 1).to(DEV).contiguous()
        R, Tm = b - a, (b + 255) // 256 * 256
        z = lambda *s: torch.full(s, float("nan"), dtype=B16, device=DEV)
        q, lat, kv, out = z(R, H, dnw + drp), z(Tm, P.dlp), z(Tm, H * (dnw + dvp) + drp), z(R, ldo)
        seq, pos = i32([1] * R), i32(list(range(a, b)))
        oq, oy, og = 0, H * (dn + dr), H * (dn + dr) + dl + dr
        nat.call("lsb_latent_expand", proj.view(-1)[oq:], proj.shape[1], proj, proj.shape[1], oy if own else -1, P.kv_norm, 1e-5, P.inv_freq, w, q, lat, kv, P.cache, P.bt, P.max_pages, page,
                 seq, pos, R, 0, b, Tm, H, dn, dnw, dr, dl, dvp, e)
        nat.call("lsb_attn_run", q, kv, Tm, i32([0]), seq, pos, i32([0]), i32([R]), proj, proj.shape[1], og, 1, out, ldo, R, H, dnw, drp, dv, dvp, 0, 0, scale)
        torch.cuda.synchronize()
        assert int(e[0]) == 0
        assert err(out[:, : H * dv], ref[a:b]) < (2e-2 if dl > 32 else 6e-2), (a, b)


@pytest.mark.parametrize("f32", [True, False])
def test_rotations_stay_exact_at_far_positions(f32):
    """Queries and rows from position 250 000 on: angles of every pair against fp64."""
    H, dn, dr, dv, dl, first, n, base = 3, 16, 32, 16, 32, 250_000, 12, 10000.0
    g = torch.Generator().manual_seed(1)
    P = Paged(H, dn, dr, dv, dl, 16, [16], f32, base)
    P.weights(torch.randn(H * dn, dl, generator=g), torch.randn(H * dv, dl, generator=g), torch.ones(dl))
    q, y = torch.randn(n, H * (dn + dr), generator=g), torch.randn(n, dl + dr, generator=g)
    P.max_pages = first // 16 + 1
    P.bt = torch.zeros(1, P.max_pages, dtype=I32, device=DEV)
    D = P.dlp + P.drp
    for rows in (n, 3):
        proj = torch.cat([q, y], 1)[:rows].to(DEV).contiguous()
        out, qn = torch.zeros(rows, H, D, dtype=P.dt, device=DEV), torch.zeros(rows, H, P.dnp, dtype=B16, device=DEV)
        pos = torch.arange(rows) + first
        e = torch.zeros(1, dtype=I32, device=DEV)
        nat.call("lsb_latent_query", proj, proj.shape[1], proj, proj.shape[1], H * (dn + dr), P.kv_norm, 1e-5, P.inv_freq, P.uk, out, qn, P.cache, P.bt, P.max_pages, 16,
                 torch.zeros(rows, dtype=I32, device=DEV), pos.to(DEV, I32), rows, H, dn, P.dnp, dr, dl, int(f32), e)
        torch.cuda.synchronize()
        tol = 1e-6 if f32 else 5e-3
        assert err(out[..., P.dlp: P.dlp + dr], O.rotate(q[:rows].view(rows, H, -1)[..., dn:].double(), pos, base)) < tol
        assert err(P.cache[0][pos % 16][:, P.dlp: P.dlp + dr], O.rotate(y[:rows, dl:].double(), pos, base)) < tol
        assert err(P.cache[0][pos % 16][:, :dl], O.rms_norm(y[:rows, :dl], 1.0, 1e-5)) < tol


# ------------------------------------------------------------------------------------------------ norms, units, router, side input
@pytest.mark.parametrize("dim", [37, 136, 1024, 2052])
@pytest.mark.parametrize("post,pre", [(2, 2), (2, 3), (0, 2), (3, 2), (2, 0), (1, 1)])
def test_residual_update_with_norms_on_both_sides(dim, post, pre):
    """0 RMS, 1 layer norm, 2 dynamic tanh, 3 none; with a dense part, expert sums as they are and weighted, and identity experts."""
    R, S, E, eps, ld = 5, 3, 4, 1e-2, (dim + 7) // 8 * 8
    g = torch.Generator().manual_seed(dim + post)
    n = lambda *s: torch.randn(*s, generator=g)
    x, sub, y, wt = n(R, dim) * 2 + 1, n(R, dim), n(R, S, ld), torch.rand(R, S, generator=g)
    ids = torch.randint(0, E + 1, (R, S), generator=g)                       # E: an identity expert
    norms = [(n(dim), n(dim), torch.tensor(0.3 + 0.4 * k)) for k in range(2)]

    def ref(kind, t, w, b, a):
        if kind == 3:
            return t
        if kind == 2:
            return O.dyt(t, a, w, b)
        c = t - t.mean(-1, keepdim=True) if kind == 1 else t
        return O.rms_norm(c, w, eps) + b

    dv = lambda kind, t: [kind] + ([None] * 3 if kind == 3 else [t[0].to(DEV), t[1].to(DEV), t[2].to(DEV) if kind == 2 else None])
    for f32 in (1, 0):
        for dense, experts in ((True, None), (False, "plain"), (True, "weighted"), (False, None)):
            resid, ds = torch.zeros(R, ld, device=DEV), torch.zeros(R, ld, device=DEV)
            resid[:, :dim], ds[:, :dim] = x.to(DEV), sub.to(DEV)
            act = torch.zeros(R, ld, dtype=F32 if f32 else B16, device=DEV)
            mo = (None, None, None, None, 0, 0, 0)
            total = sub.clone() if dense else torch.zeros(R, dim)
            if experts:
                mo = (y.to(DEV), wt.to(DEV) if experts == "weighted" else None, ids.int().to(DEV), torch.arange(E, dtype=I32, device=DEV), S, E, ld)
                val = torch.where((ids < E)[..., None], y[..., :dim], x[:, None].expand(-1, S, -1))
                total = total + ((wt[..., None] if experts == "weighted" else 1.0) * val).sum(1)
            nat.call("lsb_resid_update", act, ld, resid, ld, ds if dense else None, ld, *dv(post, norms[0]), *dv(pre, norms[1]), R, dim, eps, *mo, None, None, None, None, None, 0, 0, f32)
            want = x + ref(post, total, *norms[0])
            assert err(resid[:, :dim], want) < 2e-6, (dense, experts)
            assert err(act[:, :dim], ref(pre, want, *norms[1])) < (5e-6 if f32 else 5e-3) and float(act[:, dim:].float().abs().sum()) == 0
    out = torch.zeros(2, ld, device=DEV)
    nat.call("lsb_norm_rows", out, ld, resid, ld, i32([3, 1]), 0, norms[0][0].to(DEV), norms[0][1].to(DEV), norms[0][2].to(DEV), 2, dim, eps, 2, 1)
    assert err(out[:, :dim], O.dyt(resid[[3, 1], :dim].cpu(), norms[0][2], *norms[0][:2])) < 2e-6


@pytest.mark.parametrize("f32", [True, False])
def test_gated_units_and_the_side_gate(f32):
    R, F, ld = 7, 53, 136
    g = torch.Generator().manual_seed(2)
    z = torch.randn(R, ld, generator=g) * 3
    dz = z.to(DEV)
    for limit, alpha, shift, gated in ((0.0, 1.0, 0.0, False), (1.25, 1.702, 1.0, True), (1.25, 1.702, 1.0, False)):
        out = torch.full((R, 56), 9.0, dtype=F32 if f32 else B16, device=DEV)
        nat.call("lsb_glu", out, 56, 56, dz, ld, 3, 64, 130 if gated else -1, R, F, limit, alpha, shift, int(f32))
        a, u = z[:, 3: 3 + F], z[:, 64: 64 + F]
        if limit:
            a, u = a.clamp(max=limit), u.clamp(-limit, limit)
        want = a * torch.sigmoid(alpha * a) * (u + shift) * (torch.sigmoid(z[:, 130:131]) if gated else 1.0)
        assert err(out[:, :F], want) < (1e-6 if f32 else 5e-3) and float(out[:, F:].float().abs().sum()) == 0
    table, tok = torch.randn(20, 90, generator=g).to(B16), torch.randint(0, 20, (R,), generator=g)
    out = torch.full((R, 24), 9.0, dtype=F32 if f32 else B16, device=DEV)
    nat.call("lsb_side_gate", out, 24, dz, ld, table.to(DEV), 90, 36, 18, tok.to(DEV, I32), 20, R, int(f32))
    assert err(out[:, :18], O.gelu_tanh(z[:, :18]) * table[tok][:, 36:54].float()) < (2e-6 if f32 else 5e-3) and float(out[:, 18:].float().abs().sum()) == 0


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("R,H,F,E,top", [(3, 72, 40, 5, 2), (40, 128, 100, 6, 3), (33, 256, 128, 4, 1), (1, 256, 64, 9, 9)])
def test_experts_take_their_weight_on_the_input(R, H, F, E, top, f32):
    """Router scores as they are, clamped units, weights in front of the products; weight-streaming, tensor-core and fp32 expert kernels."""
    from layerstorm_b200.models.device_model import ExpertArena, ModelBase, MoeBuffers, QLinear, expert_layout
    g = torch.Generator().manual_seed(R + H)
    Fp = (F + 127) // 128 * 128 if H % 128 == 0 else F
    fmt = "f32" if f32 else "bf16"
    w = {f"e{e}.{k}": exactly(torch.randn(*((H, F) if k == "down" else (F, H)), generator=g) * 2 / H ** 0.5, f32) for e in range(E) for k in ("gate", "up", "down")}
    x, lg = exactly(torch.randn(R, H, generator=g), f32), torch.randn(R, E, generator=g) * 2
    arena = ExpertArena(expert_layout(fmt, H, Fp), E, E, DEV)
    dt = F32 if f32 else B16
    for e in range(E):
        pad = [torch.zeros(Fp, H), torch.zeros(Fp, H), torch.zeros(H, Fp)]
        pad[0][:F], pad[1][:F], pad[2][:, :F] = w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"]
        arena.write_expert(e, *(QLinear(fmt, t.shape[0], t.shape[1], t.to(DEV, dt)) for t in pad))
        arena.slot_of[e] = e
    z = lambda *s, dtype=F32: torch.zeros(*s, dtype=dtype, device=DEV)
    mb = MoeBuffers()
    mb.alloc_moe(z, R, top, E, E, H, Fp, tc=not f32, act_dtype=dt)
    if mb.tc_ok:
        mb.tc_xs, mb.tc_act = z(R * top, H, dtype=torch.float16), z(R * top, Fp, dtype=torch.float16)
    m = ModelBase()
    m.device, m.tp_size, m.expert_shard = torch.device(DEV), 1, "ep"
    nat.call("lsb_router_topk_grouped", lg.to(DEV), None, mb.ids, mb.wts, R, E, top, 1, 1, 0, 0, 1.0, 0, E, 1)
    ids, wt = O.route(lg, top)
    assert torch.equal(mb.ids.cpu().long(), ids) and err(mb.wts, wt) < 1e-6
    dx = x.to(DEV, dt)
    m.moe_prepare(arena, mb, dx, R, E)
    m.moe_experts(arena, mb, dx, R, E, 1.1, mb.miss, (1.702, 1.0, mb.wts))
    want = torch.stack([torch.stack([O.expert(w, f"e{i}.", (c * x[t])[None], 1.1)[0] for i, c in zip(ids[t].tolist(), wt[t])]) for t in range(R)])
    assert err(mb.y.view(R, top, H), want) < (1e-5 if f32 else 1e-2)


def test_embedding_scale():
    g = torch.Generator().manual_seed(3)
    table, tok = torch.randn(30, 40, generator=g).to(B16), torch.tensor([3, 29, 0, 31])
    f, b = torch.zeros(4, 40, device=DEV), torch.zeros(4, 40, dtype=B16, device=DEV)
    nat.call("lsb_embedding_scaled", f, b, table.to(DEV), tok.to(DEV, I32), 4, 40, 0, 30, 2.75)
    want = torch.cat([table[tok[:3]].float() * 2.75, torch.zeros(1, 40)])
    assert torch.equal(f.cpu(), want) and torch.equal(b.cpu(), want.to(B16))


# ------------------------------------------------------------------------------------------------ whole models
LONG = 200
_cache = {}


def load(tmp_path_factory, name, dtype):
    """(raw config, device model, tokens, logits of the oracle) of one geometry; models are built once.  The bf16 models have no close routing
    calls: a choice that rounding turns is no error of the kernels (routing itself is checked in fp32)."""
    key = (name, dtype, "files")
    if key not in _cache:
        c = O.MODELS[name]()
        d = tmp_path_factory.mktemp("rubasun")
        w = save_model(d, c, O.random_model(c, 11, sharp=2.0, close_calls=dtype == "float32"))
        toks = [torch.randint(0, c["vocab"], (n,), generator=torch.Generator().manual_seed(n)).tolist() for n in (LONG, 61, 97, 2)]
        wd = {k: v.double() for k, v in w.items()}
        full = [O.forward(c, wd, t, True) for t in toks]
        _cache[key] = (c, d, toks, [lg.float() for lg, _ in full], [x.float() for x in full[1][1]])
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
def test_residual_stream_after_every_layer(tmp_path_factory, name):
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


@pytest.mark.parametrize("name", ["odd", "tiles", "wide"])
def test_long_portions_match_the_oracle(tmp_path_factory, name):
    """Portions of 128 rows and more beside shorter ones, alone and with another request's tokens in the step."""
    c, m, toks, ref = load(tmp_path_factory, name, "bfloat16")
    eng = engine(m, prefill_chunk=256)
    assert sum(m._expands(b, 140, LONG) for b in m.cfg.blocks) >= 1
    for cuts in ([LONG], [140, 60], [33, 129, 38], [128, 1, 2, 69]):
        sid = eng.create_sequence()
        e = rms(feed(eng, sid, toks[0], cuts), ref[0])
        assert e < TOL["bfloat16"], (cuts, e)
        eng.free_sequence(sid)
    eng = engine(m, prefill_chunk=400)
    a, b, d, f = (eng.create_sequence() for _ in range(4))
    eng.step([Portion(d, toks[2][:3], [])])
    res = eng.step([Portion(b, toks[1][:9], [8]), Portion(a, toks[0][:150], list(range(150))), Portion(d, toks[2][3:4], [0]), Portion(f, toks[0][:130], [3, 129])],
                   return_logits=True)
    for (_, lg), want in zip(res, (ref[1][8:9], ref[0][:150], ref[2][3:4], ref[0][[3, 129]])):
        assert rms(lg, want) < TOL["bfloat16"]
    res = eng.step([Portion(a, toks[0][150:151], [0]), Portion(b, toks[1][9:10], [0]), Portion(d, toks[2][4:5], [0]), Portion(f, toks[0][130:], [0, 69])], return_logits=True)
    for (_, lg), want in zip(res, (ref[0][150:151], ref[1][9:10], ref[2][4:5], ref[0][[130, 199]])):
        assert rms(lg, want) < TOL["bfloat16"]
    _, lg = eng.prefill(b, toks[1][10:], want_logits=True)
    assert rms(lg[None], ref[1][-1:]) < TOL["bfloat16"]


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
    p = starts[0] + 57
    while p < LONG:
        _, lg = eng.decode([sids[0]], [toks[0][p]], return_logits=True)
        assert rms(lg, ref[0][p: p + 1]) < TOL[dtype], p
        p += 1


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


def test_forks_rewinds_and_hibernation_keep_the_rows(tmp_path_factory):
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


def test_layers_whose_rows_others_read_are_never_skipped(tmp_path_factory):
    c, m, toks, _ = load(tmp_path_factory, "odd", "float32")
    m.set_layer_skip([1, 2, 3])
    try:
        assert m.skip_layers == {2, 3}
        eng = engine(m)
        s = eng.create_sequence()
        lg = eng.step([Portion(s, toks[1], [60])], return_logits=True)[0][1]
        assert torch.isfinite(lg).all()
    finally:
        m.set_layer_skip([])


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
        w = {k: v.to(torch.bfloat16).float() for k, v in O.random_model(c, 11, sharp=2.0).items()}
        for p, n, r in zip(prompts, gens, reqs):
            full = list(p) + list(r.output_ids)
            lg = O.forward(c, w, full)[len(p) - 1: -1]
            best = lg.max(-1).values
            assert len(r.output_ids) == n and all(float(best[j] - lg[j, t]) < 1e-3 for j, t in enumerate(r.output_ids))
            assert eng.generate(p, n) == list(r.output_ids)
    else:
        alone = [eng.generate(p, n) for p, n in zip(prompts, gens)]
        assert sum(a == list(r.output_ids) for a, r in zip(alone, reqs)) >= 3        # ties of rounded activations may fall either way


def test_random_layers_run_and_sample():
    from layerstorm_b200.models.config import get_preset
    eng = engine(BlockModel.random_init(get_preset("tiny-rubasun"), DEV, seed=1))
    assert len(eng.generate(list(range(2, 40)), 6)) == 6 and eng.kernel_launches > 0
    s = eng.create_sequence()
    eng.prefill(s, list(range(20)))
    assert 0 <= eng.decode([s], [3], sample=(0.8, 5, 0.9, 7))[0] < 320


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
