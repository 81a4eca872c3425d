"""Fasodra without a GPU: the configuration reader, the checkpoint's names, the byte model, the distance buckets, the oracle's own mechanisms."""
import json
import math

import pytest
import torch

import fasodra_oracle as O
from gazutar_oracle import save_model
from layerstorm_b200.models.config import ModelConfig, from_hf_config, get_preset


def test_configuration_is_read_layer_by_layer_and_survives_json():
    c = O.MODELS["odd"]()
    m = from_hf_config(c)
    assert (m.architecture, m.hidden, m.vocab, m.n_layers, m.rms_eps, m.streams, m.residual_mult) == ("fasodra", 136, 301, 6, 3e-3, 3, 0.7)
    assert (m.norm_kind, m.norm_place, m.norm_topk_prob, m.logit_scale) == ("layer", "pre", True, 1.0)
    a, p, q = m.blocks[:3]
    assert (a.kind, a.heads, a.kv_heads, a.dim, a.vdim, a.chunk, a.bias_max, a.head_norm, a.half_rot, a.qkv_bias, a.window) == ("attention", 6, 2, 24, 40, 21, 50, "plain", 0, True, 0)
    assert (a.experts, a.top, a.ff, a.unit, a.correction, a.scoring) == (5, 2, 40, "relu2", False, "softmax")
    l, r = p.branches
    assert p.join == "scaled" and (l.half_rot, l.rot_base, l.head_gate, l.out_gate, l.head_norm, l.out_scale, l.chunk) == (6, 500.0, True, False, "", 0.8, 0)
    assert (r.kind, r.heads, r.dim, r.vdim, r.out_scale) == ("time_mix", 5, 12, 12, 1.2)
    l, r = q.branches
    assert q.join == "normed" and (l.half_rot, l.head_norm, l.head_gate) == (36, "weight", False)
    assert (r.kind, r.heads, r.kv_heads, r.dim, r.vdim, r.conv) == ("head_delta", 4, 2, 24, 20, 3)
    assert m.blocks[4].branches[0].out_scale == -0.6 and not m.blocks[3].has_ff
    assert [m.is_kda_layer(i) for i in range(6)] == [False, True, True, False, True, True]
    assert [len(b.mixers) for b in m.blocks] == [1, 2, 2, 1, 2, 2]
    assert ModelConfig.from_json(m.to_json()) == m
    assert from_hf_config(O.MODELS["wide"]()).streams == 5


@pytest.mark.parametrize("change", [lambda L: L[0].update(type="other"), lambda L: L[0]["mlp"].update(kind="other"), lambda L: L[1]["mixer"]["left"]["rot"].update(dims=5),
                                    lambda L: L[1]["mixer"]["left"]["rot"].update(dims=22)])
def test_configurations_that_fit_no_layer_are_refused(change):
    c = json.loads(json.dumps(O.MODELS["odd"]()))
    change(c["layers"])
    with pytest.raises(ValueError):
        from_hf_config(c)


def test_two_mixers_with_a_cache_cannot_run_side_by_side():
    m = from_hf_config(O.MODELS["odd"]())
    d = json.loads(m.to_json())
    d["blocks"][1]["branches"][1] = d["blocks"][1]["branches"][0]
    with pytest.raises(ValueError):
        ModelConfig(**d)


@pytest.mark.parametrize("name", list(O.MODELS))
def test_checkpoint_presents_every_tensor_under_the_canonical_names(tmp_path, name):
    from layerstorm_b200.models.block_model import block_weight_shapes
    from layerstorm_b200.models.checkpoint import open_checkpoint
    c = O.MODELS[name]()
    w = save_model(tmp_path, c, O.random_model(c, 1))
    cfg, ck = open_checkpoint(str(tmp_path))
    shapes = block_weight_shapes(cfg, {i: (12, 12) for i in range(cfg.n_layers)})
    assert len(shapes) == len(w) == len(ck)
    assert all(tuple(ck[k].shape) == s for k, s in shapes.items() if not k.endswith(".rel"))
    i = next(i for i, b in enumerate(cfg.blocks) if b.join == "normed" and b.branches)
    assert torch.equal(ck[f"layers.{i}.right.kda.a"], w[f"l{i}.mix.right.a"]) and torch.equal(ck[f"layers.{i}.left.out_norm"], w[f"l{i}.mix.left.out"])
    i = next(i for i, b in enumerate(cfg.blocks) if b.kind == "attention")
    assert torch.equal(ck[f"layers.{i}.attn.rel"], w[f"l{i}.mix.rel"]) and torch.equal(ck[f"layers.{i}.mix_hc.mix"], w[f"l{i}.hc1.mix"])
    assert f"layers.{i}.moe.experts.0.gate" not in ck and f"layers.{i}.left.attn.q" not in ck


def test_random_weights_cover_the_shape_and_presets_resolve():
    from layerstorm_b200.models.block_model import BlockModel, model_class
    from layerstorm_b200.models.weights import init_weights
    cfg = get_preset("tiny-fasodra")
    w = init_weights(cfg, 3)
    assert w["layers.0.attn.rel"].shape == (32, 6) and w["layers.1.right.tmix.u"].shape == (5, 24) and w["layers.3.right.kda.dt_bias"].shape == (4,)
    assert w["layers.2.ffn_hc.mix"].shape == (3, 3) and all(torch.isfinite(t).all() for t in w.values())
    assert model_class(cfg) is BlockModel and get_preset("fasodra-flash").n_moe_layers() == 8


def test_server_resolves_a_native_checkpoint_directory(tmp_path):
    from layerstorm_b200.autoconfig import sizing
    from layerstorm_b200.cli import serve
    from layerstorm_b200.config import model_config_from
    c = O.MODELS["odd"]()
    w = save_model(tmp_path, c, O.random_model(c, 1))
    args = serve.build_parser().parse_args(["--model", str(tmp_path)])
    cfg, shape, ckpt, _ = serve.resolve_config(args)
    assert shape.blocks and ckpt == str(tmp_path) and cfg["model"]["architecture"] == "fasodra" and cfg["model"]["vocab_size"] == 301
    assert model_config_from(cfg).blocks == shape.blocks
    assert sizing.kv_bytes_per_token(shape) == 2 * (2 * (32 + 64) + 2 * (32 + 32) + 3 * (64 + 32) + (64 + 32) + (32 + 32) + (64 + 32))
    assert sizing.recurrent_state_bytes_per_seq(shape) == 4 * (5 * 12 * 32 + 136 + 4 * 20 * 32 + 4 * 68 * 2 + 3 * 40 * 64 + 136 + 6 * 12 * 64 + 6 * 92 * 4)
    assert sizing.expert_slot_bytes(shape) == (2 * 136 * 128 * 2 + 4095) // 4096 * 4096
    r = sizing.resident_bytes(shape)
    mats = sum(2 * t.numel() for k, t in w.items() if ".mix." in k and t.dim() == 2 and not k.endswith((".conv", ".rel", ".u")))
    assert abs(r.attention - mats) < 0.2 * mats


@pytest.mark.parametrize("rows,reach", [(32, 200), (32, 256), (32, 128), (6, 20), (10, 9), (64, 4096), (2, 5), (12, 6 ** 3), (32, 17)])
def test_distance_buckets(rows, reach):
    """Every distance below half the rows has its own row, then the rows widen; the integer form agrees with the logarithm off the borders."""
    from layerstorm_b200.models.block_model import distance_buckets
    b = distance_buckets(rows, reach)
    half = rows // 2
    assert len(b) == reach + 1 and b[:half] == list(range(half)) and b[-1] == rows - 1 and b == sorted(b)
    for n in range(half, reach + 1):
        x = half + math.log(n / half) / math.log(reach / half) * (rows - half)
        if abs(x - round(x)) > 1e-6:
            assert b[n] == min(rows - 1, math.floor(x)), n
        else:
            assert b[n] == min(rows - 1, round(x)), n
        assert b[n] == O.bucket(n, rows, reach)
    assert O.bucket(10 * reach, rows, reach) == rows - 1
    with pytest.raises(ValueError):
        distance_buckets(rows, half)


def test_chunked_mask_and_distance_bias_pick_the_keys():
    v = O.visible(10, 4)
    assert v[5].tolist() == [False] * 4 + [True, True] + [False] * 4 and v[3, :4].all() and v.sum() == 10 + 10 + 3
    t = torch.arange(6.0)[:, None]
    b = O.distance_bias(t, 30, 20)[0]
    assert b[2, 2] == 0 and b[2, 0] == 2 and b[29, 0] == 5 and b[8, 0] in (3, 4)


def test_rotation_turns_halves_and_keeps_distances():
    x = torch.randn(12, 2, 10, dtype=torch.float64)
    y = O.rotate_half(x, 6, 50.0)
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:])
    a = 7 * 50.0 ** (-2 / 6)
    assert torch.allclose(y[7, 1, 1], x[7, 1, 1] * math.cos(a) - x[7, 1, 4] * math.sin(a)) and torch.allclose(y[7, 1, 4], x[7, 1, 4] * math.cos(a) + x[7, 1, 1] * math.sin(a))
    q, k = torch.randn(1, 1, 6, dtype=torch.float64).expand(12, 1, 6), torch.randn(1, 1, 6, dtype=torch.float64).expand(12, 1, 6)
    s = torch.einsum("ihd,jhd->ij", O.rotate_half(q, 6, 50.0), O.rotate_half(k, 6, 50.0))
    assert torch.allclose(s[9, 4], s[6, 1]) and not torch.allclose(s[9, 4], s[9, 5])


def test_time_mixing_reads_before_it_writes():
    """The current token counts through the bonus alone; the one before it without a decay of its own step."""
    r, k, v = (torch.tensor([[[1.0, 2.0]], [[3.0, 1.0]], [[1.0, 1.0]]]) for _ in range(3))
    w, u = torch.full((3, 1, 2), 0.5), torch.tensor([[10.0, 0.0]])
    o, S = O.time_mixing(r, k, v, w, u)
    assert torch.equal(o[0, 0], 10.0 * v[0, 0])
    assert torch.equal(o[1, 0], (3 * 1 + 1 * 2) * v[0, 0] + 10.0 * 9 * v[1, 0])
    assert torch.equal(S[0], 0.25 * k[0, 0][:, None] * v[0, 0] + 0.5 * k[1, 0][:, None] * v[1, 0] + k[2, 0][:, None] * v[2, 0])


def test_streams_update_from_the_old_ones_at_once():
    xs = [torch.full((1, 2), 1.0), torch.full((1, 2), 10.0)]
    mix, y = torch.tensor([[0.0, 1.0], [1.0, 0.0]]), torch.full((1, 2), 100.0)
    a, b = O.write_streams(xs, mix, torch.tensor([1.0, 2.0]), y)
    assert float(a[0, 0]) == 110.0 and float(b[0, 0]) == 201.0
