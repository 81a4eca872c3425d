"""Gazutar without a GPU: the configuration reader, the checkpoint's names, the byte model, the served step protocol on the null engine."""
import io
import json

import pytest
import torch

import gazutar_oracle as O
from layerstorm_b200.models.config import ModelConfig, from_hf_config, get_preset


def test_configuration_is_read_layer_by_layer_and_survives_json():
    c = O.MODELS["odd"]()
    m = from_hf_config(c)
    assert (m.architecture, m.hidden, m.vocab, m.n_layers, m.logit_scale, m.rms_eps, m.norm_kind) == ("gazutar", 136, 301, 5, 0.3, 3e-4, "layer")
    assert [b.kind for b in m.blocks] == ["channel_delta", "attention", "channel_delta", "attention", "attention"]
    a, d = m.blocks[1], m.blocks[0]
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.v_mix, a.scale) == (6, 2, 24, 40, 21, True, c["layers"][1]["mixer"]["scale"])
    assert (d.conv, d.experts, d.identity, d.top, d.groups, d.keep, d.ff) == (3, 5, 1, 2, 3, 2, 40)
    assert not m.blocks[2].experts and not m.is_moe_layer(2) and m.is_moe_layer(4) and m.is_kda_layer(0) and not m.is_kda_layer(1)
    assert ModelConfig.from_json(m.to_json()) == m
    with pytest.raises(ValueError):
        from_hf_config(O.model_cfg(64, 64, [{"type": "other", "mixer": {"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 8}, "mlp": None}]))


@pytest.mark.parametrize("name", list(O.MODELS))
def test_checkpoint_presents_every_tensor_under_the_canonical_names(tmp_path, name):
    from layerstorm_b200.models.block_model import block_weight_shapes
    from layerstorm_b200.models.checkpoint import open_checkpoint
    c = O.MODELS[name]()
    w = O.save_model(tmp_path, c, O.random_model(c, 1))
    cfg, ck = open_checkpoint(str(tmp_path))
    ranks = {i: (20, 23) for i in range(cfg.n_layers)}
    shapes = block_weight_shapes(cfg, ranks)
    assert len(shapes) == len(w) == len(ck)
    assert all(tuple(ck[k].shape) == s for k, s in shapes.items())
    assert torch.equal(ck["layers.0." + ("kda.q" if cfg.blocks[0].recurrent else "attn.q")], w["l0.mix.q"])
    assert "layers.0.moe.shared.0.gate" not in ck and "layers.99.mix_norm.weight" not in ck


def test_random_weights_cover_the_shape_and_presets_resolve():
    from layerstorm_b200.models.block_model import BlockModel, model_class
    from layerstorm_b200.models.device_model import DeviceModel
    from layerstorm_b200.models.weights import init_weights
    cfg = get_preset("tiny-gazutar")
    w = init_weights(cfg, 3)
    assert w["layers.1.attn.q"].shape == (6 * 32, cfg.hidden) and w["final_norm.bias"].shape == (cfg.hidden,)
    assert torch.equal(w["head.weight"], init_weights(cfg, 3)["head.weight"])
    assert model_class(cfg) is BlockModel and model_class(get_preset("tiny-mla-moe")) is DeviceModel
    assert get_preset("gazutar-flash").n_moe_layers() == 8


def test_server_resolves_a_native_checkpoint_directory(tmp_path):
    from layerstorm_b200.autoconfig import sizing
    from layerstorm_b200.cli import serve
    c = O.MODELS["tiles"]()
    O.save_model(tmp_path, c, O.random_model(c, 1))
    args = serve.build_parser().parse_args(["--model", str(tmp_path)])
    cfg, shape, ckpt, _ = serve.resolve_config(args)
    assert shape.blocks and ckpt == str(tmp_path) and cfg["model"]["architecture"] == "gazutar" and cfg["model"]["vocab_size"] == 520
    from layerstorm_b200.config import model_config_from
    assert model_config_from(cfg).blocks == shape.blocks
    assert sizing.kv_bytes_per_token(shape) == 2 * (128 + 64) + 2 * 2 * (64 + 32)
    assert sizing.recurrent_state_bytes_per_seq(shape) == 4 * (3 * (128 * 128 + 384 * 3) + 4 * (96 * 64 + 224 * 3))


def test_window_edges_and_biases_of_the_oracle():
    """The plain attention sees exactly `window` positions and takes the slope off per step back."""
    T, H = 12, 2
    q, k = torch.zeros(T, H, 4), torch.zeros(T, 1, 4)
    v = torch.eye(T)[:, None, :]
    o = O.windowed_attention(q, k, v, 1.0, 5, torch.zeros(H))
    assert torch.allclose(o[11, 0, 7:], torch.full((5,), 0.2)) and float(o[11, 0, :7].abs().sum()) == 0
    o = O.windowed_attention(q, k, v, 1.0, 0, O.slopes(2))
    r = o[6, 0, 6] / o[6, 0, 5]
    assert torch.allclose(r, torch.exp(torch.tensor(2.0 ** -4)))


def _orch(eng, **kw):
    from layerstorm_b200.serving.orchestrator import Orchestrator
    return Orchestrator(eng, eos_token_ids=[1], max_batch=4, prefill_slice_tokens=16, **kw)


@pytest.mark.parametrize("pages", [None, 14])
def test_joining_slices_ride_in_the_running_requests_steps(pages):
    """With an engine that takes mixed steps, a joining prompt's slices run in the same engine step as the running requests' tokens;
    everybody gets the tokens of being served alone, also when pages run short."""
    from layerstorm_b200.runtime.null_engine import NullEngine
    from layerstorm_b200.serving.orchestrator import InferenceRequest, Orchestrator, SamplingParams
    specs = [(20, 12), (70, 5), (33, 9), (5, 3), (48, 7)]
    prompts = [[(13 * j + 7 * i) % 250 + 4 for i in range(n)] for j, (n, _) in enumerate(specs)]

    def run(orch):
        reqs = [InferenceRequest(f"q{j}", list(p), SamplingParams(max_tokens=g, ignore_eos=True)) for j, (p, (_, g)) in enumerate(zip(prompts, specs))]
        for r in reqs:
            orch.submit_request(r)
        for _ in range(600):
            if not orch.step():
                break
        assert all(r.done.is_set() and r.error is None for r in reqs), [r.error for r in reqs]
        return [list(r.output_ids) for r in reqs]

    want = run(Orchestrator(NullEngine(vocab=300, max_seqs=16), eos_token_ids=[1]))
    eng = NullEngine(vocab=300, max_seqs=8, max_ctx=256, num_pages=pages)
    eng.supports_mixed_steps = True
    orch = _orch(eng)
    assert run(orch) == want and orch.mixed_steps > 0
    if pages is None:
        assert orch.prefill_slices > orch.mixed_steps       # the first request joined an empty batch


def test_a_failing_mixed_step_fails_every_request_in_it():
    from layerstorm_b200.runtime.null_engine import NullEngine
    from layerstorm_b200.serving.orchestrator import InferenceRequest, SamplingParams

    class Failing(NullEngine):
        def step(self, portions, return_logits=False):
            raise RuntimeError("the device said no")

    eng = Failing(vocab=300)
    eng.supports_mixed_steps = True
    orch = _orch(eng)
    a, b = (InferenceRequest(n, [5, 6, 7, 8], SamplingParams(max_tokens=20, ignore_eos=True)) for n in "ab")
    orch.submit_request(a)
    orch.step()
    orch.submit_request(b)
    for _ in range(5):
        orch.step()
    assert all("the device said no" in r.error for r in (a, b)) and not orch.running and orch.joining is None
    assert len(eng.seqs) == orch.prefix.holders()


def test_trace_replay_protocol(tmp_path):
    """Requests are admitted at their first entry, may pause, and give their slot back at the end; files hold the wanted logits in order."""
    from layerstorm_b200.cli import trace_run
    from layerstorm_b200.runtime.null_engine import NullEngine
    eng = NullEngine(vocab=64, max_seqs=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [9], "want": []}, {"id": "a", "tokens": [8], "want": [0]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "c", "tokens": [5, 6], "want": []}], "end": ["c"]},
             {"step": 3, "entries": [{"id": "b", "tokens": [4, 3], "want": [1]}, {"id": "d", "tokens": [5, 6, 7], "want": [2]}], "end": ["b", "d"]}]
    said = []
    trace_run.replay(eng, io.StringIO("\n".join(json.dumps(s) for s in steps)), str(tmp_path), said.append)
    assert said == [f"done {k}" for k in range(4)] and not eng.seqs
    rows = {k: torch.frombuffer(bytearray((tmp_path / f"{k}.f32").read_bytes()), dtype=torch.float32).view(-1, 64) for k in (0, 1, 3)}
    assert not (tmp_path / "2.f32").exists() and [len(rows[k]) for k in (0, 1, 3)] == [2, 1, 2]
    ref = NullEngine(vocab=64)
    assert torch.equal(rows[0], torch.stack([ref._logits([5]), ref._logits([5, 6, 7])])) and torch.equal(rows[1][0], ref._logits([5, 6, 7, 8]))
    assert torch.equal(rows[3], torch.stack([ref._logits([9, 4, 3]), ref._logits([5, 6, 7])]))


def test_trace_replay_tool_refuses_full_precision_for_other_model_kinds(tmp_path):
    from layerstorm_b200.cli import trace_run
    (tmp_path / "config.json").write_text(json.dumps({"model_type": "deepseek_v3", "num_hidden_layers": 2, "hidden_size": 64, "vocab_size": 64,
                                                      "num_attention_heads": 2, "kv_lora_rank": 32, "qk_nope_head_dim": 16, "v_head_dim": 16, "intermediate_size": 64}))
    assert trace_run.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"]) == 3


def test_a_family_builds_only_its_kernels():
    from layerstorm_b200 import build
    names = {p.stem for p in build._kernel_sources("blocks")}
    assert names == set(build.FAMILIES["blocks"]) and "mla" not in names and len(names) < len(build._kernel_sources())
