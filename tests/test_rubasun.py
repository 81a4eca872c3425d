"""Rubasun without a GPU: the configuration reader, the checkpoint's names, the byte model, the oracle's own mechanisms."""
import json

import pytest
import torch

import rubasun_oracle as O
from gazutar_oracle import save_model
from layerstorm_b200.models.config import ModelConfig, from_hf_config, get_preset


def test_configuration_is_read_layer_by_layer_and_survives_json():
    c = O.MODELS["odd"]()
    m = from_hf_config(c)
    assert (m.architecture, m.hidden, m.vocab, m.n_layers, m.embed_scale, m.side_dim, m.rms_eps) == ("rubasun", 136, 301, 5, 0.8, 13, 3e-2)
    assert (m.norm_kind, m.norm_place, m.logit_scale) == ("tanh", "sandwich", 1.0)
    a, b, d = m.blocks[0], m.blocks[1], m.blocks[3]
    assert (a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.kv_from, a.dense_ff, a.experts) == (6, 24, 10, 20, 40, -1, 104, 0)
    assert (b.experts, b.top, b.ff, b.limit, b.shared_ff, b.shared_limit, b.rot_base, b.scoring) == (5, 2, 40, 1.5, 72, 2.5, 500.0, "sigmoid")
    assert (b.act_alpha, b.act_shift, b.scale_input, b.correction, b.head_gate) == (1.702, 1.0, True, False, True)
    assert (d.kv_from, d.limit, d.shared_limit, d.scale) == (1, 0.7, 0.5, c["layers"][3]["mixer"]["scale"])
    assert not m.blocks[2].has_ff and a.has_ff and m.is_moe_layer(1) and not m.is_moe_layer(0) and not any(m.is_kda_layer(i) for i in range(5))
    assert ModelConfig.from_json(m.to_json()) == m
    w = from_hf_config(O.MODELS["wide"]())
    assert w.side_dim == 0 and w.blocks[0].shared_ff == 0


@pytest.mark.parametrize("change", [lambda L: L[2]["mixer"].update(kv_from=4), lambda L: L[3]["mixer"].update(kv_from=2), lambda L: L[3]["mixer"].update(kv_from=0),
                                    lambda L: L[0].update(type="other"), lambda L: L[0]["mixer"]["rot"].update(dims=4), lambda L: L[0]["mlp"].update(kind="other")])
def test_configurations_that_fit_no_layer_are_refused(change):
    c = json.loads(json.dumps(O.MODELS["odd"]()))
    change(c["layers"])
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
    assert torch.equal(ck["layers.0.attn.k_b"], w["l0.mix.uk"]) and torch.equal(ck["layers.0.mix_post_norm.alpha"], w["l0.norm1b.alpha"])
    assert "layers.1.attn.kv_a" in ck or cfg.blocks[1].kv_from >= 0
    assert "layers.0.attn.k" not in ck and "layers.99.mix_norm.weight" not in ck


def test_random_weights_cover_the_shape_and_presets_resolve():
    from layerstorm_b200.models.block_model import BlockModel, model_class
    from layerstorm_b200.models.weights import init_weights
    cfg = get_preset("tiny-rubasun")
    w = init_weights(cfg, 3)
    assert w["layers.1.attn.q"].shape == (6 * 56, cfg.hidden) and w["side_embed.weight"].shape == (cfg.vocab, 5 * 20) and w["final_norm.alpha"].shape == ()
    assert "layers.2.attn.kv_a" not in w and cfg.blocks[2].kv_from == 1
    assert model_class(cfg) is BlockModel and get_preset("rubasun-flash").n_moe_layers() == 7


def test_server_resolves_a_native_checkpoint_directory(tmp_path):
    from layerstorm_b200.autoconfig import sizing
    from layerstorm_b200.cli import serve
    from layerstorm_b200.config import model_config_from
    c = O.MODELS["odd"]()
    w = save_model(tmp_path, c, O.random_model(c, 1))
    args = serve.build_parser().parse_args(["--model", str(tmp_path)])
    cfg, shape, ckpt, _ = serve.resolve_config(args)
    assert shape.blocks and ckpt == str(tmp_path) and cfg["model"]["architecture"] == "rubasun" and cfg["model"]["vocab_size"] == 301
    assert model_config_from(cfg).blocks == shape.blocks
    assert sizing.kv_bytes_per_token(shape) == 2 * (48 + 16 + 64 + 16 + 32 + 16)            # three layers keep rows of their own
    r = sizing.resident_bytes(shape)
    of = lambda f: sum(2 * t.numel() for k, t in w.items() if f(k))
    assert r.attention == of(lambda k: ".mix." in k and not k.endswith("dkv.norm"))
    assert r.shared_expert == of(lambda k: ".shared." in k) and r.embedding == of(lambda k: k in ("embed", "side.embed"))
    assert r.dense_ffn == of(lambda k: k.partition(".")[2] in ("mlp.gate", "mlp.up", "mlp.down", "side.gate", "side.proj"))


def test_rotation_turns_adjacent_pairs_and_keeps_distances():
    x = torch.randn(3, 2, 6, dtype=torch.float64)
    p = torch.tensor([0, 7, 1000])
    y = O.rotate(x, p, 50.0)
    assert torch.equal(y[0], x[0])
    a = 7 * 50.0 ** (-2 / 6)
    u, v = x[1, 0, 2], x[1, 0, 3]
    want = torch.stack([u * torch.cos(torch.tensor(a)) - v * torch.sin(torch.tensor(a)), v * torch.cos(torch.tensor(a)) + u * torch.sin(torch.tensor(a))])
    assert torch.allclose(y[1, 0, 2:4].float(), want.float())
    q, k = torch.randn(1, 6, dtype=torch.float64), torch.randn(1, 6, dtype=torch.float64)
    dot = lambda i, j: (O.rotate(q, torch.tensor([i]), 50.0) * O.rotate(k, torch.tensor([j]), 50.0)).sum()
    assert torch.allclose(dot(40, 33), dot(1007, 1000)) and not torch.allclose(dot(40, 33), dot(40, 34))


def test_expert_input_weight_passes_through_the_nonlinear_unit():
    """Scaling an expert's input is not scaling its output: the clamp and the shifted half tell them apart."""
    g = torch.Generator().manual_seed(0)
    w = {"gate": torch.randn(8, 6, generator=g), "up": torch.randn(8, 6, generator=g), "down": torch.randn(6, 8, generator=g)}
    x = torch.randn(2, 6, generator=g)
    assert float((O.expert(w, "", 0.4 * x, 0.5) - 0.4 * O.expert(w, "", x, 0.5)).abs().max()) > 0.1
    assert torch.equal(O.expert(w, "", torch.zeros(1, 6), 0.5), torch.zeros(1, 6))
