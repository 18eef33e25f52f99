"""Lulisun through the framework's step function, cache manager and engine on a CPU (stand-in kernels), against the plain
implementation of `plain_lulisun.py`: every way of cutting the same requests gives the same logits.  And the plain
implementation's mechanisms on inputs made so that a fault would show."""

from __future__ import annotations

import json
import math

import pytest
import torch

import lulisun_configs as lc
import plain_lulisun
import replay_harness as rh
from test_kegizen_cpu import full_trace

F = torch.float64


@pytest.fixture(scope="module")
def lulisun_dirs(tmp_path_factory):
    from liteinfer_b200.weights.random_init import write_random_model

    base = tmp_path_factory.mktemp("lulisun")
    return {name: write_random_model(cfg, base / name, seed) for name, (cfg, seed, _) in lc.ALL.items()}


def expected_logits(model_dir, requests):
    config, tensors = plain_lulisun.read_model(model_dir)
    return {name: plain_lulisun.forward(config, tensors, tokens).float() for name, tokens in requests.items()}


def test_config_round_trip_and_names(lulisun_dirs):
    from liteinfer_b200.config.lulisun_config import LulisunConfig
    from liteinfer_b200.config.model_config import ConfigError
    from liteinfer_b200.config.registry import resolve

    for name, (raw, _, _) in lc.ALL.items():
        arch, config = resolve(raw)
        assert arch.name == "Lulisun" and LulisunConfig.from_dict(config.to_dict()) == config
        assert LulisunConfig.from_dict(json.loads((lulisun_dirs[name] / "config.json").read_text())) == config
    arch, config = resolve(lc.LUL_A)
    spec = arch.build_spec(config)
    assert [layer.weights_of for layer in config.layers] == [None, None, 0, 1, 0]
    assert len(spec.layers) == 2 and [entry.layer for entry in spec.schedule] == [0, 1, 0, 1, 0]
    assert all(entry.cache_of is None for entry in spec.schedule)          # every run keeps a cache of its own
    _, tensors = plain_lulisun.read_model(lulisun_dirs["lul_a"])
    assert tensors["l0.mix.left.v"].shape == (2 * 24, 64) and tensors["l0.mix.right.f.b"].shape == (36,)
    assert tensors["l0.mix.right.norm"].shape == (20,) and tensors["l0.mlp.shared.sg"].shape == (1, 64)
    assert tensors["l0.mlp.correction"].shape == (6,) and tensors["head"].shape == (211, 64)
    assert not any(n.startswith(("l2.", "l3.", "l4.")) for n in tensors)
    arch, config = resolve(lc.LUL_B)
    assert config.layers[0].left.chunk is None and config.layers[0].left.rot_dims == 0 and config.layers[1].mlp is None
    assert config.layers[0].mlp.groups == 1 and config.layers[0].mlp.shared_ff == 0
    assert [layer.block for layer in arch.build_spec(config).layers] == ["parallel_norms", "parallel_norms_mixer_only",
                                                                         "parallel_norms"]
    for path, value in ((("layers", 0, "mixer", "right", "dim"), None), (("layers", 0, "mixer", "left_scale"), None),
                        (("layers", 0, "mixer", "left", "kv_heads"), 3), (("layers", 0, "mlp", "router", "top"), 5),
                        (("layers", 0, "mlp", "router", "groups", "count"), 4), (("layers", 0, "mlp", "shared", "ff"), None),
                        (("layers", 0, "mixer", "left", "mask", "size"), 0), (("layers", 0, "mixer", "left", "rot", "dims"), 7),
                        (("norm", "eps"), None), (("layers", 2, "weights_of"), 2), (("layers", 2, "weights_of"), 9),
                        (("layers", 1, "type"), "attention"), (("layers", 1, "mlp", "kind"), "dense")):
        bad = json.loads(json.dumps(lc.LUL_A))
        at = bad
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(ConfigError):
            resolve(bad)


@pytest.mark.parametrize("name,lengths", [("lul_a", (1, 7, 61, 75)), ("lul_b", (2, 30, 45)), ("lul_c", (3, 150, 40, 18)),
                                           ("lul_d", (4, 33, 58, 21)), ("lul_e", (5, 49, 48))])
def test_all_cuts_match_plain_on_cpu(cpu_kernels, lulisun_dirs, name, lengths):
    """Whole, the tail decoded, portions down to two tokens, four live requests with pages and slots used again, every
    token a step of its own: chunks end inside prompts, at a portion's edge and among decoded tokens."""
    from liteinfer_b200.engine.loading import build_runner

    config, _, page = lc.ALL[name]
    requests = {f"r{i}": lc.prompt(config["vocab"], n, 100 + i) for i, n in enumerate(lengths)}
    expected = expected_logits(lulisun_dirs[name], requests)
    trace = full_trace(requests)
    assert trace.max_live <= 4
    runner = build_runner(lulisun_dirs[name], torch.float32, "cpu", page, -(-trace.max_tokens // page), 4)
    results = rh.run_in_process(runner, trace)
    worst, where = rh.worst_error(results, rh.gather_expected(trace, expected))
    assert worst < lc.FLOAT32_TOLERANCE[name], f"worst difference {worst} at step {where}"
    assert not runner.cache.live_requests
    for group in runner.cache.groups:
        assert group.allocator.num_held == 0


def test_layers_one_by_one_against_plain_on_cpu(cpu_kernels, lulisun_dirs):
    """The residual stream after every layer run: which layer differs first, if one does."""
    from liteinfer_b200.engine.loading import build_runner
    from liteinfer_b200.engine.runner import StepEntry

    for name in ("lul_a", "lul_b", "lul_d"):
        config, tensors = plain_lulisun.read_model(lulisun_dirs[name])
        tokens = lc.prompt(config["vocab"], 29, 3)
        want: list = []
        plain_lulisun.forward(config, tensors, tokens, want)
        runner = build_runner(lulisun_dirs[name], torch.float32, "cpu", 8, 8, 2)
        runner.cache.reserve(["a"], [29])
        context = runner.build_context([StepEntry("a", tokens, [28])])
        context.layer_trace = []
        runner.model.forward(context, runner.layer_caches)
        assert len(context.layer_trace) == len(want) == len(config["layers"])
        for stop, (got, plain) in enumerate(zip(context.layer_trace, want)):
            assert float((got.double() - plain).abs().max()) < 1e-4, f"{name}: layer {stop}"


def test_chunks_that_are_over_give_their_pages_back(cpu_kernels, lulisun_dirs):
    """However long a request grows it holds the pages of its current chunk only; the pool is smaller than the request,
    and a page is given back at the step that ends its chunk, not before."""
    from liteinfer_b200.engine.loading import build_runner
    from liteinfer_b200.engine.runner import StepEntry

    config, _, _ = lc.ALL["lul_a"]
    tokens = lc.prompt(config["vocab"], 120, 5)
    want = expected_logits(lulisun_dirs["lul_a"], {"a": tokens})["a"]
    runner = build_runner(lulisun_dirs["lul_a"], torch.float32, "cpu", 4, 12, 1)      # 48 slots a group for 120 tokens
    got = []
    for at in range(0, 120, 5):
        got.append(runner.step([StepEntry("a", tokens[at:at + 5], list(range(5)))]))
        for group in runner.cache.groups:
            chunk, total = group.need.chunk, at + 5
            first = total // chunk * chunk // 4
            assert group.allocator.num_held == max(0, -(-total // 4) - first)
            assert group.pages_at(120, 5) >= group.allocator.num_held
    assert float((torch.cat(got) - want).abs().max()) < 5e-5


def test_what_a_chunked_need_keeps():
    from liteinfer_b200.cache.manager import CacheManager
    from liteinfer_b200.parts.context import KVNeed
    from liteinfer_b200.parts.spec import ScheduleEntry

    need = KVNeed(1, 4, chunk=10)
    assert [need.first_needed(t) for t in (0, 9, 10, 11, 19, 20)] == [0, 0, 10, 10, 10, 20] and not need.keeps_all
    assert need != KVNeed(1, 4) and need != KVNeed(1, 4, window=10) and KVNeed(1, 4).keeps_all
    cache = CacheManager([(need,)], (ScheduleEntry(0),), 4, 6, 2, torch.float32, "cpu")
    for total in range(1, 41):                  # 40 tokens one by one through 24 slots, beside a request that stands still
        if total == 3:
            cache.reserve(["b"], [7])
            cache.commit("b", 7)
        cache.reserve(["a"], [total])
        cache.commit("a", total)
        cache.check_invariants()
        table = cache.block_table(0, "a")
        assert all(page < 0 for page in table[:total // 10 * 10 // 4])
        assert all(page >= 0 for page in table[total // 10 * 10 // 4:-(-total // 4)])
    assert cache.groups[0].pages_at(40, 1) <= 4 and cache.groups[0].pages_at(40, 40) == 10
    cache.release("a"); cache.release("b")
    assert cache.groups[0].allocator.num_held == 0


def test_a_slot_that_is_used_again_starts_from_zero(cpu_kernels, lulisun_dirs):
    """The memory's state of a finished request does not reach the next one in its slot."""
    from liteinfer_b200.engine.loading import build_runner
    from liteinfer_b200.engine.runner import StepEntry

    config, _, _ = lc.ALL["lul_d"]
    first, second = lc.prompt(config["vocab"], 30, 1), lc.prompt(config["vocab"], 9, 2)
    want = expected_logits(lulisun_dirs["lul_d"], {"b": second})["b"]
    runner = build_runner(lulisun_dirs["lul_d"], torch.float32, "cpu", 8, 8, 1)
    runner.step([StepEntry("a", first, [29])])
    runner.release("a")
    got = runner.step([StepEntry("b", second, list(range(9)))])
    assert float((got - want).abs().max()) < 5e-5


def test_greedy_generation_through_the_engine(cpu_kernels, lulisun_dirs):
    """`LLM.generate` (scheduler, sampler, engine loop) on a Lulisun folder picks the plain implementation's tokens."""
    from liteinfer_b200.engine.llm import LLM
    from liteinfer_b200.sampling.params import SamplingParams

    config, tensors = plain_lulisun.read_model(lulisun_dirs["lul_a"])
    prompts = [lc.prompt(config["vocab"], n, 40 + n) for n in (3, 26, 9)]
    llm = LLM(str(lulisun_dirs["lul_a"]), dtype="float32", device="cpu", block_size=16, num_gpu_blocks=32, max_num_seqs=2,
              max_model_len=64, max_num_batched_tokens=16, enable_cuda_graphs=False)
    outputs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6))
    for prompt, output in zip(prompts, outputs):
        tokens = list(prompt)
        for _ in range(6):
            tokens.append(int(plain_lulisun.forward(config, tensors, tokens)[-1].argmax()))
        assert list(output.token_ids) == tokens[len(prompt):]


# ------------------------------------------------------------- parts that another design may use
def test_side_by_side_folds_its_scales_without_a_rounding(cpu_kernels):
    """The factor left to the sum is the attention's; the memory takes the rest in its norm's 32-bit weight; with an
    attention of scale 0 its columns of the output product are zeros."""
    import liteinfer_b200.parts.model  # noqa: F401
    from liteinfer_b200.parts.registry import build_part
    from liteinfer_b200.parts.spec import PartSpec

    left = PartSpec("attention", {"hidden_size": 16, "heads": 2, "kv_heads": 1, "head_dim": 4, "v_head_dim": 6,
                                  "position": PartSpec("none", {}), "chunk": 5})
    right = PartSpec("hgrn2", {"hidden_size": 16, "heads": 1, "dim": 3, "vdim": 5, "norm_eps": 1e-5})
    for scales in ((1.5, 0.6), (0.0, 0.6), (-2.0, 0.0)):
        part = build_part("mixer", PartSpec("side_by_side", {"hidden_size": 16, "members": (left, right), "scales": scales}),
                          dtype=torch.bfloat16, device=torch.device("cpu"))
        tensors = {n: torch.ones(s.shape, dtype=torch.float32 if s.kind == "f32" else torch.bfloat16)
                   for n, s in part.tensor_specs().items()}
        part.bind(tensors)
        assert part.factor == (scales[0] or 1.0)
        assert torch.equal(part.members[1].norm_weight, torch.full((5,), scales[1] / part.factor))
        assert part.out_weight.shape == (16, 16 + 16) and part.in_weight.shape == (32 + 16, 16)     # 12 and 5 columns, 18 and 11 rows
        assert part.in_at == [(0, 18), (32, 48)] and part.out_at == [(0, 12), (16, 21)]
        assert float(part.out_weight[:, :12].float().abs().max()) == (1.0 if scales[0] else 0.0)
        assert [type(need).__name__ for need in part.cache_needs()] == ["KVNeed", "StateNeed"]


def test_a_pending_sum_holds_what_it_can():
    from liteinfer_b200 import ops

    term, rows = ops.SumTerm(torch.zeros(2, 4)), ops.RoutedRows(torch.zeros(4, 4), 2)
    both = ops.SumDelta((term,)) + ops.SumDelta((term,), rows)
    assert len(both.terms) == 2 and both.routed is rows
    with pytest.raises(ValueError):
        both + ops.SumDelta((term,))
    with pytest.raises(ValueError):
        both + ops.SumDelta((), rows)


# ------------------------------------------------------------- the plain mechanisms, on inputs that show a fault
def test_plain_chunks_on_a_planted_key():
    """One key's score stands out: every later query of its chunk finds it, the first of the next chunk does not."""
    T, D, chunk = 40, 8, 11
    g = torch.Generator().manual_seed(0)
    q = 0.01 * torch.randn(T, 2, D, generator=g, dtype=F)
    k = 0.01 * torch.randn(T, 1, D, generator=g, dtype=F)
    v = torch.randn(T, 1, 4, generator=g, dtype=F)
    for planted in (11, 16, 21):                # a chunk's first, middle and last position
        k2 = k.clone()
        k2[planted, 0] = 0.0
        k2[planted, 0, 0] = 30.0
        q[:, :, 0] = 1.0
        out = plain_lulisun.chunked_attention(q, k2, v, 1.0, chunk)
        assert torch.allclose(out[planted:22, 1], v[planted, 0].expand(22 - planted, 4), atol=1e-9)
        assert not torch.allclose(out[22, 0], v[planted, 0], atol=0.1)
        assert torch.allclose(out[22, 0], v[22, 0])         # the first of a chunk reads itself only
    whole = plain_lulisun.chunked_attention(q, k2, v, 1.0, None)
    assert torch.allclose(whole[39, 0], v[21, 0], atol=1e-9)


def test_plain_memory_keeps_and_forgets():
    """A channel whose gate is 1 keeps what it held and takes nothing; one whose gate is 0 holds the newest value only."""
    T, V = 6, 3
    v = torch.randn(T, 1, V, generator=torch.Generator().manual_seed(1), dtype=F)
    f = torch.ones(T, 1, 3, dtype=F)
    f[:, 0, 1] = 0.0
    f[:, 0, 2] = 0.5
    q = torch.eye(3, dtype=F)
    read = [plain_lulisun.forget_memory(q[c].expand(T, 1, 3), f, v)[:, 0] for c in range(3)]
    assert torch.equal(read[0], torch.zeros(T, V, dtype=F)) and torch.equal(read[1], v[:, 0])
    halves = sum(0.5 ** (T - t) * v[t, 0] for t in range(T))
    assert torch.allclose(read[2][-1], halves)
    assert float(plain_lulisun.forget_gate(torch.tensor(-50.0, dtype=F), torch.tensor(0.3, dtype=F))) == pytest.approx(0.3)
    assert float(plain_lulisun.forget_gate(torch.tensor(0.0, dtype=F), torch.tensor(0.3, dtype=F))) == pytest.approx(0.65)


def test_plain_router_chooses_by_corrected_scores_and_weighs_by_plain_ones():
    scores = torch.tensor([[0.9, 0.1, 0.5, 0.45, 0.6, 0.2]], dtype=F)            # groups (0,1) (2,3) (4,5)
    none = torch.zeros(6, dtype=F)
    router = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    chosen, weights = plain_lulisun.route_scores(scores, none, router)
    assert chosen[0].tolist() == [0, 1] and torch.allclose(weights[0], torch.tensor([0.9, 0.1], dtype=F))   # 1.0 > 0.95 > 0.8
    pulled = torch.tensor([0.0, -0.3, 0.0, 0.0, 0.0, 0.0], dtype=F)
    chosen, weights = plain_lulisun.route_scores(scores, pulled, router)
    assert chosen[0].tolist() == [2, 3] and torch.allclose(weights[0], torch.tensor([0.5, 0.45], dtype=F) / 0.95)
    chosen, _ = plain_lulisun.route_scores(scores, torch.full((6,), -5.0, dtype=F), router)     # all negative: still of the best group
    assert chosen[0].tolist() == [0, 1]
    chosen, weights = plain_lulisun.route_scores(scores, pulled * 3, {"experts": 6, "top": 3})
    assert chosen[0].tolist() == [0, 4, 2] and math.isclose(float(weights.sum()), 1.0)


def test_plain_rotation_pairs_halves_and_passes_the_rest():
    x = torch.arange(1.0, 9.0, dtype=F).view(1, 1, 8).repeat(3, 1, 1)
    turned = plain_lulisun.rotate(x, 4, 10.0)[2, 0]
    a = 2.0
    assert math.isclose(float(turned[0]), 1 * math.cos(a) - 3 * math.sin(a))
    assert math.isclose(float(turned[2]), 3 * math.cos(a) + 1 * math.sin(a))
    b = 2.0 * 10.0 ** -0.5
    assert math.isclose(float(turned[1]), 2 * math.cos(b) - 4 * math.sin(b)) and turned[4:].tolist() == [5.0, 6.0, 7.0, 8.0]
