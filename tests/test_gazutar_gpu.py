"""Gazutar on the device against the plain evaluation in gazutar_oracle.py: every mechanism alone, then whole models of several geometries
through the engine - prompts, decoding, portions, mixed batches, reused pages and slots, generation through the server's scheduler."""
import pytest
import torch

pytestmark = pytest.mark.gpu

import gazutar_oracle as O
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

    def run(self, parts, wq=None, wk=None, mix=0, lam=None, vfirst=None, window=0, scale=1.0, slope=None, gate=True, NS=1, run_rows=None, eps=1e-5):
        """parts: (sequence, first position, q [n, H dk], k [n, G dk], v [n, G dv], gate [n, H dv])."""
        H, G, dk, dv = self.H, self.G, self.dk, self.dv
        rows = [torch.cat([q, k, v, gt], 1) for _, _, q, k, v, gt in parts]
        proj = torch.cat(rows).float().to(DEV).contiguous()
        R = proj.shape[0]
        seq = i32([s for s, p0, q, *_ in parts for _ in range(len(q))])
        pos = i32([p0 + j for s, p0, q, *_ in parts for j in range(len(q))])
        n = [len(p[2]) for p in parts]
        row0 = i32([sum(n[:j]) for j in range(len(n))])
        q = torch.zeros(R, H, self.dkp, dtype=self.dt, device=DEV)
        out = torch.zeros(R, H * dv + 8, dtype=self.dt, device=DEV)
        op, ml = torch.zeros(R * H * NS * self.dvp, device=DEV), torch.zeros(R * H * NS * 2, device=DEV)
        oq, ok, ov, og = 0, H * dk, (H + G) * dk, (H + G) * dk + G * dv
        nat.call("lsb_attn_prep", proj, proj.shape[1], oq, ok, ov, wq, wk, eps, vfirst, mix, lam, q, self.cache, self.bt, self.max_pages, seq, pos, R, H, G,
                 dk, dv, self.dkp, self.dvp, self.page, int(self.f32))
        nat.call("lsb_attn", q, self.cache, self.bt, self.max_pages, self.page, seq, pos, row0, i32(n), len(n), run_rows or max(n), proj, proj.shape[1],
                 og if gate else -1, out, H * dv + 8, op, ml, NS, R, H, G, dk, dv, self.dkp, self.dvp, window, scale, slope, 0, 0, None, 0, 1.0, None, 1, int(self.f32))
        torch.cuda.synchronize()
        return out[:, : H * dv].float().cpu()


GEOMETRIES = [(4, 2, 32, 32), (6, 1, 24, 40), (8, 2, 64, 64), (3, 3, 128, 96), (20, 1, 64, 128), (2, 1, 200, 256), (2, 2, 20, 272)]


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,G,dk,dv", GEOMETRIES)
def test_attention_sees_far_keys_and_exactly_its_window(H, G, dk, dv, f32):
    """One key stands out for every query: the token itself, one at a page border, the last one inside the window or the first one outside it
    (then a nearer decoy must win).  Prompt runs of unequal length, then single rows with and without key splits."""
    if f32 and (H, G) not in ((6, 1), (3, 3)):
        pytest.skip("the CUDA-core kernel has one form")
    T, W, page = 150, 37, 16
    g = torch.Generator().manual_seed(H * 100 + dk)
    r = (lambda t: t) if f32 else (lambda t: t.to(B16).float())
    lens = [T, T - 29]
    data = []
    for n in lens:
        k = torch.nn.functional.normalize(torch.randn(n, G, dk, generator=g), dim=-1) * dk ** 0.5
        v = torch.randn(n, G, dv, generator=g)
        q = torch.empty(n, H, dk)
        for i in range(n):
            for h in range(H):
                back = (0, W - 1, W, i - i // page * page, i - max(0, i // page * page - 1), 1)[(i + h) % 6]
                q[i, h] = 40.0 / dk * k[max(0, i - back), h // (H // G)] + (0.0 if back < W else 12.0 / dk * k[i, h // (H // G)])
        data.append((r(q.reshape(n, -1)), r(k.reshape(n, -1)), r(v.reshape(n, -1)), torch.randn(n, H * dv, generator=g)))
    slope = O.slopes(H)
    for window, bias in ((W, True), (0, False)):
        sl = slope if bias else torch.zeros(H)
        ref = [O.windowed_attention(q.view(-1, H, dk), k.view(-1, G, dk), v.view(-1, G, dv), 0.9, window, sl).reshape(len(q), -1) * torch.sigmoid(gt)
               for q, k, v, gt in data]
        kw = dict(window=window, scale=0.9, slope=slope.to(DEV) if bias else None)
        tol = 2e-5 if f32 else 8e-3
        P = Paged(H, G, dk, dv, page, lens, f32)
        cut = lambda s, a, b: (s, a, *(t[a:b] for t in data[s]))
        out = P.run([cut(0, 0, T), cut(1, 0, 3)], **kw)
        assert err(out, torch.cat([ref[0], ref[1][:3]])) < tol
        out = P.run([cut(1, 3, 70)], **kw)
        assert err(out, ref[1][3:70]) < tol
        for a in range(70, lens[1]):                                     # decoded
            for NS in ((1, 3) if a % 10 == 0 else (1,)):
                assert err(P.run([cut(1, a, a + 1)], NS=NS, **kw), ref[1][a: a + 1]) < tol, (a, NS)
        P = Paged(H, G, dk, dv, page, lens, f32, seed=9)
        outs = [P.run([cut(0, a, a + 2), cut(1, a, a + 2)], NS=1 + a // 2 % 2, **kw) for a in range(0, 120, 2)]
        assert err(torch.cat([o[:2] for o in outs]), ref[0][:120]) < tol and err(torch.cat([o[2:] for o in outs]), ref[1][:120]) < tol


@pytest.mark.parametrize("f32", [True, False])
def test_projection_norms_value_mixing_and_gate(f32):
    H, G, dk, dv, n, eps = 6, 2, 24, 40, 33, 1e-3
    g = torch.Generator().manual_seed(3)
    q, k, v1, v2 = (torch.randn(n, w, generator=g) * 3 for w in (H * dk, G * dk, G * dv, G * dv))
    gt = torch.randn(n, H * dv, generator=g)
    wq, wk, lam = 1 + 0.3 * torch.randn(H * dk, generator=g), 1 + 0.3 * torch.randn(G * dk, generator=g), torch.tensor(0.35)
    vf = torch.full((n, G * dv), 99.0, device=DEV)
    qn, kn = O.rms_norm(q, wq, eps).view(n, H, dk), O.rms_norm(k, wk, eps).view(n, G, dk)
    kw = dict(wq=wq.to(DEV), wk=wk.to(DEV), eps=eps, scale=0.4, window=9, slope=O.slopes(H).to(DEV), vfirst=vf, lam=lam.to(DEV))
    for mix, v, used, gate in ((1, v1, v1, True), (2, v2, O.mix_values(v2, v1, lam), True), (2, v1, v1, False)):
        ref = O.windowed_attention(qn, kn, used.view(n, G, dv), 0.4, 9, O.slopes(H)).reshape(n, -1)
        out = Paged(H, G, dk, dv, 16, [n], f32).run([(0, 0, q, k, v, gt)], mix=mix, gate=gate, **kw)
        assert err(out, ref * torch.sigmoid(gt) if gate else ref) < (3e-5 if f32 else 1e-2), mix
    assert torch.equal(vf.cpu(), v1)


# ------------------------------------------------------------------------------------------------ delta rule
class Delta:
    def __init__(self, H, G, dk, dv, taps, ra=12, rg=20, f32=True, seed=0, slots=3, mode=0):
        g = torch.Generator().manual_seed(seed)
        n = lambda *s: torch.randn(*s, generator=g)
        self.s = dict(H=H, G=G, dk=dk, dv=dv, taps=taps)
        self.f32, self.mode, self.ra, self.rg = f32, mode, (ra + 7) // 8 * 8, (rg + 7) // 8 * 8
        r = (lambda t: t) if f32 else (lambda t: t.to(B16).float())
        self.w_a, self.w_g = r(n(H * dk, ra) / ra ** 0.5), r(n(H * dv, rg) / rg ** 0.5)
        self.conv = [torch.rand(c, taps, generator=g) * 2 - 1 for c in (G * dk, G * dk, H * dv)]
        self.a_log, self.dt, self.onorm = torch.rand(H, generator=g) * 4 - 3.5, torch.rand(H * dk, generator=g) * 3 - 3, 1 + 0.2 * n(dv)
        al = lambda x: (x + 7) // 8 * 8
        self.widths = [G * dk, G * dk, H * dv, H, ra, rg]
        self.offs = [sum(al(x) for x in self.widths[:j]) for j in range(6)]
        self.ld = sum(al(x) for x in self.widths)
        pad = lambda t, c: torch.nn.functional.pad(t, (0, c - t.shape[1])).to(F32 if f32 else B16).to(DEV).contiguous()
        self.da, self.dg = pad(self.w_a, self.ra), pad(self.w_g, self.rg)
        self.da2, self.dg2 = torch.cat([self.da] * 2, 1).contiguous(), torch.cat([self.dg] * 2, 1).contiguous()
        self.state = torch.zeros(slots, H, dv, nat.call("lsb_delta_key_pad", dk), device=DEV)
        self.hist = torch.zeros(slots, H, 2 * dk + dv, taps - 1, device=DEV)
        self.dconv = [c.to(DEV) for c in self.conv]
        self.vec = [t.to(DEV) for t in (torch.exp(self.a_log), self.dt, self.onorm)]

    def inputs(self, T, seed):
        g = torch.Generator().manual_seed(seed)
        return [torch.randn(T, w, generator=g) for w in self.widths]

    def reference(self, x, eps=1e-5):
        s = self.s
        H, G, dk, dv = s["H"], s["G"], s["dk"], s["dv"]
        T = x[0].shape[0]
        q, k, v = (O.short_conv(x[j].double(), self.conv[j].double()) for j in range(3))
        q, k = O.unit(q.view(T, G, dk)) * dk ** -0.5, O.unit(k.view(T, G, dk))
        q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
        a = (x[4].double() @ self.w_a.double().T + self.dt).view(T, H, dk)
        A = torch.exp(self.a_log.double())[None, :, None]
        gl = -A * O.softplus(a) if self.mode == 0 else -4.0 * torch.sigmoid(A * a)
        o, S = O.delta_rule(q, k, v.view(T, H, dv), torch.exp(gl), torch.sigmoid(x[3].double()))
        o = O.rms_norm(o, self.onorm.double(), eps).reshape(T, -1) * torch.sigmoid(x[5].double() @ self.w_g.double().T)
        return o.float(), S.float()

    def run(self, parts, form, eps=1e-5):
        """parts: (slot, inputs rows); form: few | rows | chunk (rows with the chunk-parallel recurrence from 16 rows on)."""
        s = self.s
        H, G, dk, dv = s["H"], s["G"], s["dk"], s["dv"]
        n = [p[1][0].shape[0] for p in parts]
        R = sum(n)
        proj = torch.zeros(R, self.ld, device=DEV)
        r0 = 0
        for (_, x), m in zip(parts, n):
            for o, t in zip(self.offs, x):
                proj[r0: r0 + m, o: o + t.shape[1]] = t.to(DEV)
            r0 += m
        out = torch.zeros(R, H * dv + 4, dtype=F32 if self.f32 else B16, device=DEV)
        long_min = 16
        longs = [m for m in n if m >= long_min] if form == "chunk" else []
        chunks = sum((m + 63) // 64 for m in longs)
        scratch = torch.full((nat.call("lsb_delta_scratch_floats", R, H, dk, dv, self.ra, self.rg),), float("nan"), device=DEV)
        cw = torch.full((max(1, nat.call("lsb_delta_chunk_floats", chunks, H, dk)),), float("nan"), device=DEV)
        e = torch.zeros(1, dtype=I32, device=DEV)
        nat.call("lsb_delta_forward", proj, self.ld, *self.offs, self.ra, self.rg, self.da, self.dg, None if self.f32 else self.da2, None if self.f32 else self.dg2,
                 *self.dconv, *self.vec, self.state, self.hist, i32([sum(n[:j]) for j in range(len(n))]), i32(n), i32([p[0] for p in parts]), out,
                 H * dv + 4, len(n), R, H, G, dk, dv, s["taps"], self.mode, dk ** -0.5, -4.0, eps, int(self.f32), int(form == "few"), scratch,
                 len(n) - len(longs), len(longs), chunks, long_min, cw, e)
        torch.cuda.synchronize()
        assert int(e[0]) == 0
        return out[:, : H * dv].float().cpu()


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,G,dk,dv,taps", [(4, 2, 32, 64, 4), (3, 3, 24, 20, 3), (2, 1, 48, 96, 1), (6, 2, 64, 40, 2), (2, 2, 128, 128, 4), (2, 1, 100, 130, 5),
                                            (1, 1, 160, 72, 4), (3, 1, 20, 256, 6)])
def test_delta_rule_forms_agree_with_the_recurrence(H, G, dk, dv, taps, f32):
    """Whole runs token by token and chunk-parallel, a cut in every short length, and the one-kernel form, on interleaved state slots."""
    T = 170
    tol = 3e-5 if f32 else 1e-2
    forms = ["rows"] + (["chunk"] if dk <= 128 else []) + (["few"] if dv <= nat.call("lsb_delta_few_max_dv", dk) else [])
    for form in forms:
        D = Delta(H, G, dk, dv, taps, f32=f32, seed=dk)
        a, b = D.inputs(T, 1), D.inputs(T, 2)
        (ra, Sa), (rb, _) = D.reference(a), D.reference(b)
        sl = lambda x, i, j: [t[i:j] for t in x]
        pos_a = pos_b = 0
        cuts = [(1, 2), (2, 1), (40, 70), (7, 1), (64, 3), (1, 93), (55, 0)] if form != "few" else [(1, 1), (2, 3), (8, 1)] * 14
        for na, nb in cuts:
            parts = [(2, sl(a, pos_a, pos_a + na))] + ([(0, sl(b, pos_b, pos_b + nb))] if nb else [])
            out = D.run(parts, form)
            assert err(out[:na], ra[pos_a: pos_a + na]) < tol, (form, pos_a, na)
            assert nb == 0 or err(out[na:], rb[pos_b: pos_b + nb]) < tol, (form, pos_b, nb)
            pos_a, pos_b = pos_a + na, pos_b + nb
        if pos_a == T:
            assert err(D.state[2, ..., :dk].transpose(1, 2), Sa) < (3e-5 if f32 else 3e-3)
        assert float(D.state[1].abs().max()) == 0 and float(D.state[..., dk:].abs().sum()) == 0 and float(D.hist[1].abs().sum()) == 0


@pytest.mark.parametrize("form", ["few", "rows", "chunk"])
def test_delta_rule_with_the_bounded_decay(form):
    D = Delta(2, 1, 32, 32, 4, seed=5, mode=1)
    x = D.inputs(96 if form != "few" else 8, 7)
    assert err(D.run([(0, x)], form), D.reference(x)[0]) < 3e-5


def test_delta_rule_survives_strong_and_weak_decays():
    """Decay factors from ~1 to exactly 0 inside one chunk: the chunk form works on logarithms and stays finite."""
    D = Delta(2, 2, 32, 32, 4, seed=6)
    D.vec[0].copy_(torch.tensor([60.0, 1e-4]))
    D.a_log = torch.log(torch.tensor([60.0, 1e-4]))
    x = D.inputs(150, 8)
    ref = D.reference(x)[0]
    outs = {f: Delta.run(D, [(s, x)], f) for s, f in enumerate(("rows", "chunk"))}
    assert all(torch.isfinite(o).all() and err(o, ref) < 3e-5 for o in outs.values())


# ------------------------------------------------------------------------------------------------ norms, router, experts
@pytest.mark.parametrize("layer,bias", [(1, True), (1, False), (0, False)])
@pytest.mark.parametrize("dim", [37, 136, 1024])
def test_post_norm_update_and_gathered_norm_rows(layer, bias, dim):
    R, eps, ld = 5, 1e-2, (dim + 7) // 8 * 8
    g = torch.Generator().manual_seed(dim)
    x, sub = torch.randn(R, dim, generator=g) * 4 + 3, torch.randn(R, dim, generator=g) * 0.3 + 2
    w, b = torch.randn(dim, generator=g), torch.randn(dim, generator=g) if bias else torch.zeros(dim)
    nrm = lambda t: O.layer_norm(t, w, b, eps) if layer else O.rms_norm(t, w, eps)
    for f32 in (1, 0):
        resid, ds = torch.zeros(R, ld, device=DEV), torch.zeros(R, ld, device=DEV)
        resid[:, :dim], ds[:, :dim] = x.to(DEV), sub.to(DEV)
        act = torch.zeros(R, ld, dtype=F32 if f32 else B16, device=DEV)
        nat.call("lsb_resid_update", act, ld, resid, ld, ds, ld, layer, w.to(DEV), b.to(DEV) if bias else None, None, 3, None, None, None, R, dim, eps, None, None,
                 None, None, 0, 0, 0, None, None, None, None, None, 0, 0, f32)
        want = x + nrm(sub)
        assert err(resid[:, :dim], want) < 1e-6 and err(act[:, :dim], want) < (1e-6 if f32 else 5e-3) and float(act[:, dim:].float().abs().sum()) == 0
        out = torch.zeros(3, ld, dtype=act.dtype, device=DEV)
        nat.call("lsb_norm_rows", out, ld, resid, ld, i32([4, 0, 4]), 0, w.to(DEV), b.to(DEV) if bias else None, None, 3, dim, eps, layer, f32)
        assert err(out[:, :dim], nrm(want[[4, 0, 4]])) < (1e-5 if f32 else 5e-3)
        nat.call("lsb_norm_rows", out, ld, resid, ld, None, 2, w.to(DEV), b.to(DEV) if bias else None, None, 3, dim, eps, layer, f32)
        assert err(out[:, :dim], nrm(want[2:5])) < (1e-5 if f32 else 5e-3)


@pytest.mark.parametrize("E,ident,top,count,keep", [(8, 2, 3, 2, 1), (6, 0, 4, 1, 1), (4, 4, 2, 8, 3), (5, 1, 2, 3, 2), (60, 4, 8, 8, 4)])
def test_grouped_router_and_identity_experts(E, ident, top, count, keep):
    """Negative choice scores, best-score groups, weights without the correction; identity outputs add the residual itself."""
    R, n, H = 40, E + ident, 72
    g = torch.Generator().manual_seed(E)
    lg, corr = torch.randn(R, n, generator=g) * 2, -2 + 0.4 * torch.randn(n, generator=g)
    ids, wt = O.route({"experts": E, "top": top, "groups": {"count": count, "keep": keep}}, lg, corr)
    di, dw = torch.zeros(R, top, dtype=I32, device=DEV), torch.zeros(R, top, device=DEV)
    nat.call("lsb_router_topk_grouped", lg.to(DEV), corr.to(DEV), di, dw, R, n, top, count, keep, 1, 0, 1.0, 0, n, 1)
    assert torch.equal(di.cpu().long(), ids) and err(dw, wt) < 1e-5
    y, x = torch.randn(R, top, H, generator=g), torch.randn(R, H, generator=g)
    w, b = torch.randn(H, generator=g), torch.randn(H, generator=g)
    val = torch.where((ids < E)[..., None], y, x[:, None, :].expand(-1, top, -1))
    want = x + O.layer_norm((wt[..., None] * val).sum(1), w, b, 1e-5)
    resid, act = x.to(DEV).contiguous(), torch.zeros(R, H, device=DEV)
    nat.call("lsb_resid_update", act, H, resid, H, None, 0, 1, w.to(DEV), b.to(DEV), None, 3, None, None, None, R, H, 1e-5, y.to(DEV), dw, di,
             torch.arange(E, dtype=I32, device=DEV), top, E, H, None, None, None, None, None, 0, 0, 1)
    assert err(resid, want) < 1e-5 and torch.equal(resid, act)


# ------------------------------------------------------------------------------------------------ whole models
LONG = 200
_cache = {}


def load(tmp_path_factory, name, dtype):
    """(raw config, device model, tokens, logits of the oracle) of one geometry; models are built once.  The bf16 models have no close
    routing calls: a choice that rounding turns is no error of the kernels (routing itself is checked in fp32)."""
    key = (name, dtype, "files")
    if key not in _cache:
        c = O.MODELS[name]()
        d = tmp_path_factory.mktemp("gazutar")
        w = O.save_model(d, c, O.random_model(c, 11, sharp=2.0, close_calls=dtype == "float32"))
        toks = [torch.randint(0, c["vocab"], (n,), generator=torch.Generator().manual_seed(n)).tolist() for n in (LONG, 61, 97, 2)]
        wd = {k: v.double() for k, v in w.items()}
        _cache[key] = (c, d, toks, [O.forward(c, wd, t).float() for t in toks])
    c, d, toks, ref = _cache[key]
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(O.MODELS))
def test_prompts_portions_and_decoding_match_the_oracle(tmp_path_factory, name, dtype):
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


def test_a_step_larger_than_a_pass_and_wrong_portions(tmp_path_factory):
    c, m, toks, ref = load(tmp_path_factory, "odd", "float32")
    eng = engine(m, prefill_chunk=32)
    a, b, d = (eng.create_sequence() for _ in range(3))
    eng.step([Portion(b, toks[1][:1], [])])
    res = eng.step([Portion(a, toks[0], [0, 70, LONG - 1]), Portion(b, toks[1][1:2], [0]), Portion(d, toks[2], list(range(97)))], return_logits=True)
    assert rms(res[0][1], ref[0][[0, 70, LONG - 1]]) < 2e-4 and rms(res[1][1], ref[1][1:2]) < 2e-4 and rms(res[2][1], ref[2]) < 2e-4
    for bad in ([], [Portion(a, [], [])], [Portion(a, [1], [1])], [Portion(a, [1]), Portion(a, [2])]):
        with pytest.raises(ValueError):
            eng.step(bad)


def test_running_out_of_pages_fails_before_anything_is_committed(tmp_path_factory):
    from layerstorm_b200.runtime.engine import KvPoolExhausted
    c, m, toks, ref = load(tmp_path_factory, "odd", "float32")
    eng = engine(m, num_pages=6)
    a, b = eng.create_sequence(), eng.create_sequence()
    eng.step([Portion(a, toks[0][:40], [])])
    with pytest.raises(KvPoolExhausted):
        eng.step([Portion(a, toks[0][40:41], [0]), Portion(b, toks[2][:90], [])])
    assert eng.seq_len(a) == 40 and eng.seq_len(b) == 0
    eng.free_sequence(b)
    assert rms(eng.step([Portion(a, toks[0][40:60], [19])], return_logits=True)[0][1], ref[0][59:60]) < 2e-4


@pytest.mark.parametrize("name,dtype", [("tiles", "bfloat16"), ("attention first", "float32")])
def test_long_decoding_through_the_captured_step(tmp_path_factory, name, dtype):
    """Three sequences decode together far beyond every window."""
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


def test_forks_anchored_rewinds_and_hibernation_keep_the_state(tmp_path_factory):
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
        w = {k: v for k, v in O.random_model(c, 11, sharp=2.0).items()}
        w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
        for p, n, r in zip(prompts, gens, reqs):
            full = list(p) + list(r.output_ids)
            lg = O.forward(c, w, full)[len(p) - 1: -1]
            best = lg.max(-1).values
            assert len(r.output_ids) == n and all(float(best[j] - lg[j, t]) < 1e-3 for j, t in enumerate(r.output_ids))
            assert eng.generate(p, n) == list(r.output_ids)
    else:
        alone = [eng.generate(p, n) for p, n in zip(prompts, gens)]
        assert sum(a == list(r.output_ids) for a, r in zip(alone, reqs)) >= 3        # ties of rounded activations may fall either way


def test_sampling_and_confidence_run_on_the_device(tmp_path_factory):
    c, m, toks, ref = load(tmp_path_factory, "tiles", "bfloat16")
    eng = engine(m)
    s = eng.create_sequence()
    eng.prefill(s, toks[0][:20])
    t = eng.decode([s], [toks[0][20]], sample=(0.8, 5, 0.9, 7))[0]
    assert int((ref[0][20] > ref[0][20][t]).sum()) < 12
    _, conf = eng.decode([s], [toks[0][21]], confidence=True)
    assert 0 < conf[0][0] <= 1


def test_random_full_size_layers_run():
    from layerstorm_b200.models.config import get_preset
    eng = engine(BlockModel.random_init(get_preset("tiny-gazutar"), DEV, seed=1))
    out = eng.generate(list(range(2, 40)), 6)
    assert len(out) == 6 and eng.kernel_launches > 0


def test_the_server_boots_a_checkpoint_directory(tmp_path_factory):
    from layerstorm_b200.cli import serve
    c, m, toks, ref = load(tmp_path_factory, "odd", "bfloat16")
    d = _cache["odd", "bfloat16", "files"][1]
    args = serve.build_parser().parse_args(["--model", str(d), "--max-sequence-length", "512", "--max-concurrent", "3", "--tokenizer-mode", "byte"])
    cfg, shape, ckpt, _ = serve.resolve_config(args)
    eng = serve.build_engine(cfg, shape, ckpt, args)
    assert isinstance(eng.model, BlockModel) and eng.supports_mixed_steps and eng.model.kv_fmt == "bf16"
    s = eng.create_sequence()
    _, lg = eng.prefill(s, toks[1], want_logits=True)
    assert rms(lg[None], ref[1][-1:]) < TOL["bfloat16"]
