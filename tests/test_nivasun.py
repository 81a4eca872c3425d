"""Nivasun without a GPU: the configuration reader, the checkpoint's names, the byte model, the staged previous tokens, the oracle's own mechanisms."""
import json
import math

import pytest
import torch

import nivasun_oracle as O
from gazutar_oracle import save_model
from layerstorm_b200.models.config import ModelConfig, from_hf_config, get_preset


def test_configuration_is_read_layer_by_layer_and_survives_json():
    m = from_hf_config(O.MODELS["odd"]())
    assert (m.architecture, m.hidden, m.vocab, m.n_layers, m.rms_eps, m.input_conv, m.softcap, m.embed_scale) == ("nivasun", 136, 301, 5, 3e-3, 4, 9.0, 3.0)
    assert (m.norm_kind, m.norm_place, m.norm_scalar, m.norm_topk_prob, m.loop, m.bigram) == ("rms", "parallel", True, True, [1, 3, 2], [97, 1000003, 12345])
    l, a, d = m.blocks[:3]
    assert (l.kind, l.heads, l.dim, l.vdim, l.kv_rank, l.q_rank, l.rot_dim, l.window, l.out_gate, l.head_gate) == ("latent_attention", 5, 20, 12, 44, 36, 0, 33, True, False)
    assert (a.kind, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.half_rot, a.pair_rot, a.rot_base) == ("attention", 6, 2, 24, 24, 21, 10, 0, 500.0)
    assert a.shared_kv and a.temp and a.sink and a.maps == 1 and not d.shared_kv and not d.sink
    assert (d.kind, d.maps, d.diff, d.half_rot, d.pair_rot, d.rot_base, d.window, d.vdim) == ("attention", 2, 0.35, 0, 12, 300.0, 26, 36)
    assert (a.experts, a.top, a.ff, a.shared_ff, a.logit_bias, a.correction, a.unit, a.act_alpha, a.limit) == (7, 3, 24, 40, True, False, "glu", 1.0, 0.0)
    assert not d.has_ff and not any(m.is_kda_layer(i) for i in range(5)) and m.keeps_state
    assert m.layer_runs() == [(0, -1), (1, 0), (2, -1), (1, 1), (2, -1), (3, -1), (4, -1)]
    assert ModelConfig.from_json(m.to_json()) == m
    assert from_hf_config(O.MODELS["tiles"]()).layer_runs() == [(0, 0), (1, -1), (0, 1), (1, -1), (2, -1), (3, -1)]
    one = from_hf_config(O.MODELS["ones"]())
    assert one.layer_runs() == [(0, 0), (1, -1), (2, -1), (3, -1)] and not one.keeps_state
    assert [[i, -1 if t is None else t] for i, t in O.layer_runs(O.MODELS["wide"]())] == [list(r) for r in from_hf_config(O.MODELS["wide"]()).layer_runs()]


@pytest.mark.parametrize("change", [lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="other"), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=5),
                                    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), lambda c: c["layers"][1]["mixer"].update(vdim=20), lambda c: c["loop"].update(stop=6),
                                    lambda c: c["loop"].update(start=3), lambda c: c["loop"].update(times=0)])
def test_configurations_that_fit_no_layer_are_refused(change):
    c = json.loads(json.dumps(O.MODELS["odd"]()))
    change(c)
    with pytest.raises(ValueError):
        from_hf_config(c)


@pytest.mark.parametrize("name", list(O.MODELS))
def test_checkpoint_presents_every_tensor_under_the_canonical_names(tmp_path, name):
    from layerstorm_b200.models.block_model import block_weight_shapes
    from layerstorm_b200.models.checkpoint import open_checkpoint
    c = O.MODELS[name]()
    w = save_model(tmp_path, c, O.random_model(c, 1))
    cfg, ck = open_checkpoint(str(tmp_path))
    shapes = block_weight_shapes(cfg)
    assert len(shapes) == len(w) == len(ck)
    assert all(tuple(ck[k].shape) == s for k, s in shapes.items())
    for i, b in enumerate(cfg.blocks):
        p, q = f"layers.{i}.attn.", f"l{i}.mix."
        for k, n in {"latent_attention": [("q_a", "dq"), ("q_b", "uq"), ("kv_a_norm", "dkv.norm"), ("k_b", "uk"), ("g", "g")]}.get(b.kind, [("lq2", "lq2"), ("v", "v")] if b.maps > 1 else [("temp", "temp"), ("sink", "sink")]):
            assert torch.equal(ck[p + k], w[q + n])
    assert torch.equal(ck["loop_step"], w["loop.step"]) and torch.equal(ck["bigram.weight"], w["bigram"]) and torch.equal(ck["layers.0.input_conv"], w["l0.canon1"])
    assert torch.equal(ck["layers.0.moe.router_bias"], w["l0.mlp.router.b"]) and torch.equal(ck["layers.0.moe.shared.0.up"], w["l0.mlp.shared.up"])
    assert "layers.0.ffn_norm.weight" not in ck


def test_random_weights_cover_the_shape_and_presets_resolve():
    from layerstorm_b200.models.block_model import BlockModel, model_class
    from layerstorm_b200.models.weights import init_weights
    cfg = get_preset("tiny-nivasun")
    w = init_weights(cfg, 3)
    assert w["bigram.weight"].shape == (510, 192) and w["loop_step"].shape == (2, 192) and w["layers.0.mix_norm.weight"].shape == () and w["layers.2.attn.q"].shape == (128, 192)
    assert all(torch.isfinite(t).all() for t in w.values()) and "layers.0.attn.v" not in w
    assert model_class(cfg) is BlockModel and len(get_preset("nivasun-flash").layer_runs()) == 9


def test_server_resolves_a_native_checkpoint_directory(tmp_path):
    from layerstorm_b200.autoconfig import sizing
    from layerstorm_b200.cli import serve
    from layerstorm_b200.config import model_config_from
    c = O.MODELS["odd"]()
    w = save_model(tmp_path, c, O.random_model(c, 1))
    args = serve.build_parser().parse_args(["--model", str(tmp_path)])
    cfg, shape, ckpt, _ = serve.resolve_config(args)
    assert shape.blocks and ckpt == str(tmp_path) and cfg["model"]["architecture"] == "nivasun" and cfg["model"]["vocab_size"] == 301
    assert model_config_from(cfg).blocks == shape.blocks and model_config_from(cfg).loop == shape.loop
    # layers in the loop hold a cache and a state per pass
    assert sizing.kv_bytes_per_token(shape) == 2 * (48 + 2 * (2 * (32 + 32) + 3 * (2 * 32 + 64)) + 3 * (64 + 64) + (2 * 32 + 32))
    assert sizing.recurrent_state_bytes_per_seq(shape) == 7 * 3 * 136 * 4
    r = sizing.resident_bytes(shape)
    mats = sum(2 * t.numel() for k, t in w.items() if ".mix." in k and t.dim() == 2)
    assert abs(r.attention - mats) < 0.05 * mats
    assert r.embedding == (301 + 98) * 136 * 2


def test_a_tool_compiles_the_files_of_the_mixers_that_a_model_has():
    from layerstorm_b200 import build
    fam = {n: build.family_of(get_preset(n)) for n in ("tiny-nivasun", "tiny-rubasun", "tiny-fasodra", "tiny-gazutar", "tiny-mla-moe")}
    assert list(fam.values()) == ["blocks_latent", "blocks_latent", "blocks_delta_tmix", "blocks_delta", None]
    assert {p.stem for p in build._kernel_sources("blocks_latent")} == set(build.FAMILIES["blocks"]) | {"latent"}


def test_the_previous_token_is_staged_with_the_step():
    """In front of a run's first row stands the sequence's last token, in front of a sequence's first token nothing."""
    from types import SimpleNamespace

    from layerstorm_b200.runtime.engine import Engine, SequenceState
    m = SimpleNamespace(cfg=from_hf_config(O.MODELS["odd"]()), device=torch.device("cpu"), V_local=301)
    eng = object.__new__(Engine)
    eng.cfg, eng.row_tier, eng.h2d_bytes = m.cfg, None, 0
    eng.seqs = {0: SequenceState(0, 3, [], [7, 8, 9]), 2: SequenceState(2), 3: SequenceState(3, 1, [], [40])}
    rows = [(1, 0, 3), (2, 0, 4), (30, 2, 0), (31, 2, 1), (32, 2, 2), (50, 3, 1)]
    seen = {}

    class Rows:
        R = 8
        inp = torch.zeros(10, 8, dtype=torch.int32)
        prev_tok = inp[9]
        h_ring, h_ev, h_i = [torch.zeros(10, 8, dtype=torch.int32)], [None], 0
    ws = Rows()
    ws.h_ring, ws.h_ev = ws.h_ring * 4, [None] * 4
    ev = SimpleNamespace(record=lambda s: None)
    orig = torch.cuda.Event, torch.cuda.current_stream
    torch.cuda.Event, torch.cuda.current_stream = (lambda: ev), (lambda: None)
    try:
        eng._stage(ws, rows, [(0, 2, 0), (2, 3, 2), (5, 1, 3)])
    finally:
        torch.cuda.Event, torch.cuda.current_stream = orig
    assert ws.prev_tok[:6].tolist() == [9, 1, -1, 30, 31, 40] and ws.inp[0, :6].tolist() == [1, 2, 30, 31, 32, 50]


# ------------------------------------------------------------------------------------------------ the oracle's mechanisms
def test_bigram_rows_and_the_first_token():
    assert O.bigram_rows([5, 6, 2], 10, 3, 7) == [10, (15 + 42) % 10, (18 + 14) % 10]
    c = {"embedding": {"scale": 2.0, "bigram": {"buckets": 2, "mul_prev": 1, "mul_cur": 0}}}
    w = {"embed": torch.arange(6.0)[:, None], "bigram": torch.tensor([[100.0], [200.0], [300.0]])}
    assert O.embed(c, w, [3, 4, 5]).flatten().tolist() == [6.0 + 300.0, 8.0 + 200.0, 10.0 + 100.0]


def test_input_conv_weighs_the_current_token_last():
    h = torch.tensor([[1.0], [10.0], [100.0]])
    assert O.input_conv(h, torch.tensor([[1.0, 2.0, 3.0]])).flatten().tolist() == [3.0, 32.0, 321.0]
    assert O.input_conv(h, torch.tensor([[3.0]])).flatten().tolist() == [3.0, 30.0, 300.0]


def test_window_sink_and_temperature():
    v = O.visible(6, 3)
    assert v[5].tolist() == [False] * 3 + [True] * 3 and v[1].tolist() == [True, True] + [False] * 4 and v.sum() == 15
    s = torch.full((2, 1, 4), float("-inf"))
    s[:, 0, 1:] = torch.tensor([0.0, 1.0, 2.0])
    p = O.softmax_with_sink(s, torch.tensor([0.5, 80.0]))
    z = sum(math.exp(x) for x in (0.0, 1.0, 2.0, 0.5))
    assert torch.allclose(p[0, 0], torch.tensor([0.0, 1 / z, math.e / z, math.e ** 2 / z])) and 0 < float(p[1].sum()) < 1e-30
    q, k = torch.randn(4, 2, 3), torch.randn(4, 1, 3)
    a = O.attend(q, k, k, 0.7, 4, torch.tensor([1.0, 3.0]))
    assert torch.allclose(a[:, 0], O.attend(q, k, k, 0.7, 4)[:, 0]) and torch.allclose(a[:, 1], O.attend(q, k, k, 2.1, 4)[:, 1], atol=1e-6)


def test_rotations_pair_halves_or_neighbours():
    x = torch.randn(12, 2, 10, dtype=torch.float64)
    a = 7 * 50.0 ** (-2 / 6)
    y, z = O.rotate_half(x, 6, 50.0), O.rotate_pairs(x, 6, 50.0)
    assert torch.equal(y[0], x[0]) and torch.equal(z[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:]) and torch.equal(z[..., 6:], x[..., 6:])
    assert torch.allclose(y[7, 1, 1], x[7, 1, 1] * math.cos(a) - x[7, 1, 4] * math.sin(a)) and torch.allclose(y[7, 1, 4], x[7, 1, 4] * math.cos(a) + x[7, 1, 1] * math.sin(a))
    assert torch.allclose(z[7, 1, 2], x[7, 1, 2] * math.cos(a) - x[7, 1, 3] * math.sin(a)) and torch.allclose(z[7, 1, 3], x[7, 1, 3] * math.cos(a) + x[7, 1, 2] * math.sin(a))


def test_differential_attention_subtracts_the_second_map():
    """A second map equal to the first leaves (1 - lambda) of it in front of the norm, whose sign is all that remains of the factor."""
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 3, "scale": 1.0, "diff": 0.25, "mask": {"size": 9}, "rot": {"base": 10.0, "dims": 2}}
    w = {k: torch.zeros(2) for k in ("lq1", "lk1", "lq2", "lk2")} | {"q": torch.zeros(4, 2), "k": torch.zeros(4, 2), "v": torch.randn(3, 2), "o": torch.eye(3)}
    assert float(O.map_weight(m, w, "")) == 0.25
    h = torch.randn(1, 2)
    want = 0.75 * O.rms(h @ w["v"].T, 0.0)
    assert torch.allclose(O.differential_mixer(m, 0.0, w, "", h), want, atol=1e-6)
    w |= {"lq1": torch.tensor([1.0, 0.5]), "lk1": torch.tensor([1.0, 1.0])}
    assert math.isclose(float(O.map_weight(m, w, "")), math.exp(1.5) - 1 + 0.25, rel_tol=1e-6)
    assert torch.allclose(O.differential_mixer(m, 0.0, w, "", h), -want, atol=1e-6)


def test_router_weights_are_the_softmax_of_the_chosen():
    ids, wt = O.route(torch.tensor([[1.0, 3.0, -2.0, 2.0]]), 2)
    assert ids.tolist() == [[1, 3]] and torch.allclose(wt, torch.tensor([[math.e, 1.0]]) / (1 + math.e))
