"""Sogazen through the framework's step function, cache manager and engine on a CPU (stand-in kernels), against the plain
implementation of `plain_sogazen.py`: every way of cutting the same requests gives the same logits.  And the plain
implementation's mechanisms on inputs made so that a fault would show."""

from __future__ import annotations

import json
import math

import pytest
import torch

import plain_sogazen
import replay_harness as rh
import sogazen_configs as sc
from test_kegizen_cpu import full_trace

F = torch.float64


@pytest.fixture(scope="module")
def sogazen_dirs(tmp_path_factory):
    base = tmp_path_factory.mktemp("sogazen")
    return {name: sc.write_model(cfg, base / name, seed) for name, (cfg, seed, _) in sc.ALL.items()}


def expected_logits(model_dir, requests):
    config, tensors = plain_sogazen.read_model(model_dir)
    return {name: plain_sogazen.forward(config, tensors, tokens).float() for name, tokens in requests.items()}


def test_config_round_trip_and_names(sogazen_dirs):
    from liteinfer_b200.config.model_config import ConfigError
    from liteinfer_b200.config.registry import resolve
    from liteinfer_b200.config.sogazen_config import SogazenConfig

    for name, (raw, _, _) in sc.ALL.items():
        arch, config = resolve(raw)
        assert arch.name == "Sogazen" and SogazenConfig.from_dict(config.to_dict()) == config
        assert SogazenConfig.from_dict(json.loads((sogazen_dirs[name] / "config.json").read_text())) == config
    _, tensors = plain_sogazen.read_model(sogazen_dirs["sog_a"])
    assert tensors["l0.mix.left.q.b"].shape == (96,) and tensors["l0.mix.left.k.norm"].shape == (32,)
    assert "l0.mix.left.v" not in tensors and tensors["l0.mix.right.in"].shape == (2 * 48 + 2 * 2 * 20 + 4, 64)
    assert tensors["l0.mix.right.conv"].shape == (48 + 80, 3) and tensors["l0.mix.left.out"].shape == (64,)
    assert tensors["l1.mix.w1"].shape == (12, 64) and tensors["l1.mix.u"].shape == (3, 20)
    assert tensors["l1.mlp.router"].shape == (5, 64) and "l1.mlp.e3.up" not in tensors and "l1.mlp.e0.gate" not in tensors
    assert tensors["head"].shape == (211, 64)
    arch, config = resolve(sc.SOG_B)
    assert config.logit_softcap == 0.0 and config.layers[1].left.softcap == 0.0 and config.layers[1].left.rot_dims == 0
    assert config.layers[0].mlp.identity == 0 and config.layers[1].mlp is None and config.layers[3].mixer.decay_rank is None
    assert [layer.block for layer in arch.build_spec(config).layers] == ["output_norm", "output_norm_mixer_only", "output_norm",
                                                                         "output_norm_mixer_only"]
    for path, value in ((("layers", 0, "mixer", "right", "state"), None), (("layers", 0, "mixer", "left", "scale"), None),
                        (("layers", 0, "mixer", "left", "kv_heads"), 4), (("layers", 0, "mixer", "left", "vdim"), 24),
                        (("layers", 0, "mixer", "right", "groups"), 3), (("layers", 0, "mixer", "right", "norm_groups"), 5),
                        (("layers", 0, "mixer", "left", "rot", "dims"), 7), (("layers", 0, "mixer", "right", "conv"), 0),
                        (("layers", 0, "mlp", "limit"), None), (("layers", 0, "mlp", "limit"), 0.0),
                        (("layers", 1, "mlp", "router", "top"), 6), (("layers", 1, "mlp", "expert", "ff"), None),
                        (("layers", 1, "mixer", "dim"), None), (("layers", 1, "type"), "delta"), (("norm", "eps"), None),
                        (("layers", 0, "mlp", "kind"), "sparse"), (("logit_softcap",), -1.0)):
        with pytest.raises(ConfigError):
            resolve(sc.changed(sc.SOG_A, path, value))


def test_the_decays_inner_width_is_the_checkpoints(cpu_kernels, sogazen_dirs, tmp_path):
    """config.json need not name it, and two tensors that do not fit each other are refused."""
    from safetensors.torch import load_file, save_file

    from liteinfer_b200.weights.loader import WeightsError, load_model

    raw = json.loads((sogazen_dirs["sog_a"] / "config.json").read_text())
    del raw["layers"][1]["mixer"]["decay_rank"]
    (tmp_path / "config.json").write_text(json.dumps(raw))
    tensors = load_file(str(sogazen_dirs["sog_a"] / "model.safetensors"))
    save_file(tensors, str(tmp_path / "model.safetensors"))
    model, _ = load_model(tmp_path, torch.float32, "cpu")
    assert model.layers[1].parts["mixer"].w1.shape == (12, 64)
    save_file({**tensors, "l1.mix.w1": tensors["l1.mix.w1"][:7].clone()}, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError):
        load_model(tmp_path, torch.float32, "cpu")
    save_file({**tensors, "l1.mix.w1": tensors["l1.mix.w1"][:, :60].clone()}, str(tmp_path / "model.safetensors"))
    with pytest.raises(WeightsError):
        load_model(tmp_path, torch.float32, "cpu")


@pytest.mark.parametrize("name,lengths", [("sog_a", (1, 7, 61, 75)), ("sog_b", (2, 30, 45)), ("sog_c", (3, 70, 40, 18)),
                                           ("sog_d", (4, 33, 58, 21)), ("sog_e", (5, 49, 48))])
def test_all_cuts_match_plain_on_cpu(cpu_kernels, sogazen_dirs, name, lengths):
    """Whole, the tail decoded, portions down to two tokens, four live requests with pages and slots used again, every
    token a step of its own."""
    from liteinfer_b200.engine.loading import build_runner

    config, _, page = sc.ALL[name]
    requests = {f"r{i}": sc.prompt(config["vocab"], n, 100 + i) for i, n in enumerate(lengths)}
    expected = expected_logits(sogazen_dirs[name], requests)
    trace = full_trace(requests)
    assert trace.max_live <= 4
    runner = build_runner(sogazen_dirs[name], torch.float32, "cpu", page, -(-trace.max_tokens // page), 4)
    results = rh.run_in_process(runner, trace)
    worst, where = rh.worst_error(results, rh.gather_expected(trace, expected))
    assert worst < sc.FLOAT32_TOLERANCE[name], f"worst difference {worst} at step {where}"
    assert not runner.cache.live_requests
    for group in runner.cache.groups:
        assert group.allocator.num_held == 0


def test_layers_one_by_one_against_plain_on_cpu(cpu_kernels, sogazen_dirs):
    """The residual stream after every layer: which layer differs first, if one does."""
    from liteinfer_b200.engine.loading import build_runner
    from liteinfer_b200.engine.runner import StepEntry

    for name in ("sog_a", "sog_b", "sog_d"):
        config, tensors = plain_sogazen.read_model(sogazen_dirs[name])
        tokens = sc.prompt(config["vocab"], 29, 3)
        want: list = []
        plain_sogazen.forward(config, tensors, tokens, want)
        runner = build_runner(sogazen_dirs[name], torch.float32, "cpu", 8, 8, 2)
        runner.cache.reserve(["a"], [29])
        context = runner.build_context([StepEntry("a", tokens, [28])])
        context.layer_trace = []
        runner.model.forward(context, runner.layer_caches)
        assert len(context.layer_trace) == len(want) == len(config["layers"])
        for stop, (got, plain) in enumerate(zip(context.layer_trace, want)):
            assert float((got.double() - plain).abs().max()) < 1e-4, f"{name}: layer {stop}"


def test_a_slot_that_is_used_again_starts_from_zero(cpu_kernels, sogazen_dirs):
    """Memories, convolution tails and last tokens of a finished request do not reach the next one in its slot."""
    from liteinfer_b200.engine.loading import build_runner
    from liteinfer_b200.engine.runner import StepEntry

    for name in ("sog_a", "sog_d"):
        config, _, _ = sc.ALL[name]
        first, second = sc.prompt(config["vocab"], 30, 1), sc.prompt(config["vocab"], 9, 2)
        want = expected_logits(sogazen_dirs[name], {"b": second})["b"]
        runner = build_runner(sogazen_dirs[name], torch.float32, "cpu", 8, 8, 1)
        runner.step([StepEntry("a", first, [29])])
        runner.release("a")
        got = runner.step([StepEntry("b", second, list(range(9)))])
        assert float((got - want).abs().max()) < 1e-4


def test_greedy_generation_through_the_engine(cpu_kernels, sogazen_dirs):
    """`LLM.generate` (scheduler, sampler, engine loop) on a Sogazen folder picks the plain implementation's tokens."""
    from liteinfer_b200.engine.llm import LLM
    from liteinfer_b200.sampling.params import SamplingParams

    config, tensors = plain_sogazen.read_model(sogazen_dirs["sog_a"])
    prompts = [sc.prompt(config["vocab"], n, 40 + n) for n in (3, 26, 9)]
    llm = LLM(str(sogazen_dirs["sog_a"]), dtype="float32", device="cpu", block_size=16, num_gpu_blocks=32, max_num_seqs=2,
              max_model_len=64, max_num_batched_tokens=16, enable_cuda_graphs=False)
    outputs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6))
    for prompt, output in zip(prompts, outputs):
        tokens = list(prompt)
        for _ in range(6):
            tokens.append(int(plain_sogazen.forward(config, tensors, tokens)[-1].argmax()))
        assert list(output.token_ids) == tokens[len(prompt):]


def test_parts_refuse_what_they_cannot_do():
    import liteinfer_b200.parts.model  # noqa: F401
    from liteinfer_b200.parts.registry import build_part
    from liteinfer_b200.parts.spec import PartSpec

    where = dict(dtype=torch.float32, device=torch.device("cpu"))
    attention = {"hidden_size": 16, "heads": 2, "kv_heads": 1, "head_dim": 4, "position": PartSpec("none", {}),
                 "values_are_keys": True, "qk_norm": "projection", "bias": True, "out_bias": False}
    built = build_part("mixer", PartSpec("attention", attention), **where)
    assert built.joint_norm and not built.has_biases and set(built.tensor_specs()) == {
        "q_proj.weight", "k_proj.weight", "o_proj.weight", "q_proj.bias", "k_proj.bias", "q_norm.weight", "k_norm.weight"}
    for options in ({"qk_norm": "head"}, {"v_head_dim": 8}, {"head_gate": True}, {"sink": True, "fixed_sink": 0.0}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("attention", {**attention, **options}), **where)
    moe = {"hidden_size": 16, "intermediate_size": 8, "experts": 4, "top": 2, "activation": "relu_squared", "gives_sum": True,
           "identity": 3}
    assert build_part("feed_forward", PartSpec("routed_experts", moe), **where).tensor_specs()["router.weight"].shape == (7, 16)
    for options in ({"gives_sum": False}, {"groups": 2}, {"top": 8}, {"identity": -1}, {"activation": "relu"}):
        with pytest.raises(ValueError):
            build_part("feed_forward", PartSpec("routed_experts", {**moe, **options}), **where)
    with pytest.raises(ValueError):
        build_part("feed_forward", PartSpec("gated_mlp", {"hidden_size": 16, "intermediate_size": 8,
                                                          "activation": "capped_swiglu"}), **where)


# ------------------------------------------------------------- the plain mechanisms, on inputs that show a fault
def test_plain_attention_on_a_planted_key_and_on_silence():
    """One key's score stands out: every later query finds it however far away; a query whose scores are far below 0 reads
    nothing; with equal scores of 0 over n keys each weighs 1 / (n + 1); a cap bounds the score."""
    T, D = 60, 8
    g = torch.Generator().manual_seed(0)
    q = 0.01 * torch.randn(T, 2, D, generator=g, dtype=F)
    k = 0.01 * torch.randn(T, 1, D, generator=g, dtype=F)
    v = torch.randn(T, 1, 4, generator=g, dtype=F)
    q[:, :, 0] = 1.0
    for planted in (0, 7, 40):
        k2 = k.clone()
        k2[planted, 0, 0] = 40.0
        out = plain_sogazen.quiet_attention(q, k2, v, 1.0, None)
        assert torch.allclose(out[planted:, 1], v[planted, 0].expand(T - planted, 4), atol=1e-9)
        if planted:
            assert not torch.allclose(out[planted - 1, 0], v[planted, 0], atol=0.1)
    low = k.clone()
    low[:, 0, 0] = -50.0
    assert float(plain_sogazen.quiet_attention(q, low, v, 1.0, None).abs().max()) < 1e-15
    flat = plain_sogazen.quiet_attention(torch.zeros_like(q), k, v, 1.0, 5.0)
    assert torch.allclose(flat[9, 0], v[:10, 0].sum(0) / 11)
    capped = plain_sogazen.quiet_attention(q, k2, v, 1.0, 2.0)           # one key at exp(2), 59 about exp(0), the sink
    assert torch.allclose(capped[59, 0], (v[:, 0].sum(0) + (math.e ** 2 - 1) * v[40, 0]) / (math.e ** 2 + 60), atol=2e-2)


def test_plain_values_are_the_keys_before_norm_and_rotation():
    mixer = {"heads": 1, "kv_heads": 1, "dim": 4, "vdim": 4, "scale": 0.0, "rot": {"dims": 4, "base": 10.0}}
    w = {"q": torch.eye(4, dtype=F), "k": 2.0 * torch.eye(4, dtype=F), "o": torch.eye(4, dtype=F)}
    w.update({n + ".b": torch.arange(4, dtype=F) for n in "qk"})
    w.update({n + ".norm": torch.full((4,), 7.0, dtype=F) for n in "qk"})
    h = torch.randn(3, 4, generator=torch.Generator().manual_seed(1), dtype=F)
    got = plain_sogazen.left_mixer(h, w, "", mixer, 1e-6)
    keys = 2.0 * h + torch.arange(4, dtype=F)
    assert torch.allclose(got[2], keys.sum(0) / 4)          # scores of 0: each of three keys weighs 1 / (3 + 1)


def test_plain_state_space_keeps_and_forgets():
    """No decay: a sum of what was written; one that is large: the token's own alone; the group of a head is its neighbours'."""
    T, V = 5, 3
    x = torch.randn(T, 2, V, generator=torch.Generator().manual_seed(1), dtype=F)
    b = torch.zeros(T, 2, 2, dtype=F)
    b[:, 0, 0] = 1.0
    b[:, 1, 1] = 2.0
    c = torch.ones(T, 2, 2, dtype=F)
    dt = torch.full((T, 2), 0.5, dtype=F)
    a_log = torch.tensor([-60.0, 60.0], dtype=F)
    y = plain_sogazen.state_space(x, b, c, dt, a_log, torch.tensor([0.0, 10.0], dtype=F))
    assert torch.allclose(y[:, 0], 0.5 * x[:, 0].cumsum(0)) and torch.allclose(y[:, 1], (0.5 * 2.0 + 10.0) * x[:, 1])
    z = torch.zeros(T, 6, dtype=F)
    flat = plain_sogazen.gated_group_norm(y.reshape(T, 6), z + 1.0, torch.ones(6, dtype=F), 2, 1e-12)
    assert torch.allclose(flat.view(T, 2, 3).pow(2).mean(-1), torch.ones(T, 2, dtype=F))
    assert float(plain_sogazen.softplus(torch.tensor(0.0, dtype=F))) == pytest.approx(math.log(2))
    taps = torch.tensor([[0.0, 1.0], [1.0, 0.0]], dtype=F)
    moved = plain_sogazen.causal_conv(torch.arange(8, dtype=F).view(4, 2), taps, torch.tensor([0.5, 0.0], dtype=F))
    assert moved.tolist() == [[0.5, 0.0], [2.5, 1.0], [4.5, 3.0], [6.5, 5.0]]       # the last tap is the token's own


def test_plain_memory_reads_before_it_writes():
    """The token's own key and value are seen through the bonus only; what was written before, through the decays since."""
    T, D = 4, 2
    r, k = torch.ones(T, 1, D, dtype=F), torch.ones(T, 1, D, dtype=F)
    v = torch.randn(T, 1, D, generator=torch.Generator().manual_seed(2), dtype=F)
    decay = torch.tensor([1.0, 0.5], dtype=F).expand(T, 1, D)
    none = plain_sogazen.bonus_memory(r, k, v, decay, torch.zeros(1, D, dtype=F))[:, 0]
    assert torch.equal(none[0], torch.zeros(D, dtype=F)) and torch.allclose(none[1], 2.0 * v[0, 0])
    assert torch.allclose(none[3], (1 + 0.25) * v[0, 0] + (1 + 0.5) * v[1, 0] + 2.0 * v[2, 0])
    some = plain_sogazen.bonus_memory(r, k, v, decay, torch.tensor([[3.0, 4.0]], dtype=F))[:, 0]
    assert torch.allclose(some, none + 7.0 * v[:, 0])
    h = torch.arange(6.0, dtype=F).view(3, 2)
    assert plain_sogazen.token_shift(h, torch.tensor([1.0, 0.0], dtype=F)).tolist() == [[0.0, 1.0], [0.0, 3.0], [2.0, 5.0]]


def test_plain_router_chooses_by_corrected_scores_and_identity_experts_give_back():
    logits = torch.log(torch.tensor([[0.4, 0.3, 0.2, 0.1]], dtype=F))
    chosen, weights = plain_sogazen.route(logits, torch.zeros(4, dtype=F), 2)
    assert chosen[0].tolist() == [0, 1] and torch.allclose(weights[0], torch.tensor([0.4, 0.3], dtype=F))
    chosen, weights = plain_sogazen.route(logits, torch.tensor([-0.5, 0.0, 0.0, 0.4], dtype=F), 2)
    assert chosen[0].tolist() == [3, 1] and torch.allclose(weights[0], torch.tensor([0.1, 0.3], dtype=F))
    w = {"router": torch.zeros(3, 2, dtype=F), "correction": torch.tensor([0.0, 1.0, 1.0], dtype=F),
         "e0.up": torch.ones(1, 2, dtype=F), "e0.down": torch.ones(2, 1, dtype=F)}
    h = torch.tensor([[1.0, -4.0], [2.0, 3.0]], dtype=F)
    mlp = {"router": {"experts": 1, "identity": 2, "top": 2}}
    assert torch.allclose(plain_sogazen.moe_ff(h, w, "", mlp), h * (2.0 / 3.0))
    w["correction"][0] = 2.0
    got = plain_sogazen.moe_ff(h, w, "", mlp)                # the expert (relu, squared) and one identity, a third each
    assert torch.allclose(got, h / 3.0 + torch.tensor([[0.0], [25.0]], dtype=F) / 3.0)


def test_plain_capped_gate():
    g, u = torch.tensor([5.0, -3.0, 0.5], dtype=F), torch.tensor([-9.0, 9.0, 0.25], dtype=F)
    s = lambda x: 1.0 / (1.0 + math.exp(-1.702 * x))
    want = [2.0 * s(2.0) * -1.0, -3.0 * s(-3.0) * 3.0, 0.5 * s(0.5) * 1.25]
    assert plain_sogazen.capped_gate(g, u, 2.0).tolist() == pytest.approx(want)


def test_plain_rotation_pairs_halves_and_passes_the_rest():
    x = torch.arange(1.0, 9.0, dtype=F).view(1, 1, 8).repeat(3, 1, 1)
    turned = plain_sogazen.rotate(x, 4, 10.0)[2, 0]
    a, b = 2.0, 2.0 * 10.0 ** -0.5
    assert math.isclose(float(turned[0]), 1 * math.cos(a) - 3 * math.sin(a))
    assert math.isclose(float(turned[2]), 3 * math.cos(a) + 1 * math.sin(a))
    assert math.isclose(float(turned[1]), 2 * math.cos(b) - 4 * math.sin(b)) and turned[4:].tolist() == [5.0, 6.0, 7.0, 8.0]
