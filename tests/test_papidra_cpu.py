"""Papidra on the CPU path (fp32) against the plain statement in ``papidra_oracle``: configuration, loader, layers, cache and
state manager, batching, prefix cache, speculation and generation."""
import pytest
import torch

import papidra_cases as PC
import papidra_oracle as O
from atlas_b200.config import EngineConfig, ModelConfig
from atlas_b200.engine import LLMEngine
from atlas_b200.loader.load import load_model
from atlas_b200.replay import build_engine
from atlas_b200.sampling import SamplingParams

TOL = 2e-4


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    root = tmp_path_factory.mktemp("papidra")
    made = {}

    def get(name):
        if name not in made:
            path = str(root / name)
            made[name] = (path,) + PC.write(path, name)
        return made[name]
    return get


@pytest.mark.parametrize("name", list(PC.CASES))
def test_logits_and_every_layer_match_the_plain_statement(folder, name):
    path, cfg, w = folder(name)
    toks = PC.tokens(cfg, 70, 1)
    layers = []
    want = O.forward(cfg, w, toks, layers)
    model = load_model(path, dtype="float32", max_pos=128)
    model.capture_layers = tuple(range(len(model.layers)))
    got = model.forward_dense_reference(toks)
    for i, (a, b) in enumerate(zip(model.aux_hidden, layers)):
        assert (a - b).abs().max() < TOL * b.abs().max(), f"layer {i}"
    assert PC.spread(got, want) < TOL


@pytest.mark.parametrize("cuts", [[2], [1], [3, 16, 1, 7], [24], [23, 2], [64]], ids=str)
def test_logits_do_not_depend_on_the_cut(folder, cuts):
    path, cfg, w = folder("mixed")
    toks = PC.tokens(cfg, 75, 2)
    eng = build_engine(path, "float32", 128, device="cpu")
    got = PC.feed_alone(eng, "a", toks, PC.portions(75, cuts))
    assert PC.spread(got, O.forward(cfg, w, toks)) < TOL
    assert eng.pool.num_free == eng.pool.num_blocks and eng.state_pool.num_free == eng.state_pool.num_slots


def test_unequal_batches_on_reused_pages_and_slots(folder):
    path, cfg, w = folder("mixed")
    eng = build_engine(path, "float32", 256, device="cpu")
    plans = {"a": (PC.tokens(cfg, 60, 3), PC.portions(60, [17, 1, 1, 2]), 0), "b": (PC.tokens(cfg, 5, 4), [1] * 5, 0),
             "c": (PC.tokens(cfg, 90, 5), PC.portions(90, [2, 33, 1]), 1), "d": (PC.tokens(cfg, 31, 6), [31], 3)}
    first = PC.feed_together(eng, plans)
    # the second round starts in another order, so every request sits on pages and a slot that others used before
    second = PC.feed_together(eng, {r: plans[r] for r in ("d", "c", "b", "a")})
    for r, (toks, _, _) in plans.items():
        want = O.forward(cfg, w, toks)
        assert PC.spread(first[r], want) < TOL and PC.spread(second[r], want) < TOL
    eng.pool.check_invariants()


def test_feed_refuses_more_than_the_pools_hold(folder):
    path, cfg, _ = folder("ones")
    eng = build_engine(path, "float32", 64, device="cpu")
    with pytest.raises(ValueError):
        eng.feed([("a", [cfg["vocab"]], [0])])
    for i in range(4):
        eng.feed([(f"r{i}", PC.tokens(cfg, 16, i), [])])
    with pytest.raises(RuntimeError):
        eng.feed([("r4", [1], [0])])
    with pytest.raises(RuntimeError):
        eng.feed([("r0", [1], [0])])                     # every page is taken


def test_generation_prefix_cache_and_preemption(folder):
    """Greedy generation through the scheduler equals the plain statement's greedy continuation: alone, in a batch, from a
    cached prefix (state snapshots) and with so few pages that sequences are preempted."""
    path, cfg, w = folder("mixed")
    prompts = [PC.tokens(cfg, n, 10 + n) for n in (40, 9, 33)]
    prompts.append(prompts[0][:35] + PC.tokens(cfg, 6, 99))

    def greedy(p, n):
        p = list(p)
        for _ in range(n):
            p.append(int(O.forward(cfg, w, p)[-1].argmax()))
        return p[-n:]
    want = [greedy(p, 6) for p in prompts]
    sp = SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True)
    for kw in ({}, {"max_prefill_tokens": 16}, {"num_kv_blocks": 7, "admission_watermark_tokens": 0},
               {"ngram_speculative": True, "num_drafts": 3, "mtp_gate": False}):
        base = {"num_kv_blocks": 64, "max_num_seqs": 4, "max_seq_len": 96, "ssm_checkpoint_interval": 16}
        eng = LLMEngine(load_model(path, dtype="float32", max_pos=128), EngineConfig(**{**base, **kw}))
        for _ in range(2):
            assert [o.output_tokens for o in eng.generate(prompts, sp)] == want, kw
        if not kw:
            assert eng.radix.stats.hit_tokens > 0


def test_rejected_drafts_leave_the_state_alone(folder):
    """A verify step scores drafts without moving the recurrent state; committing n rows equals having fed n tokens."""
    from atlas_b200.models import ForwardBatch
    path, cfg, w = folder("mixed")
    model = load_model(path, dtype="float32", max_pos=128)
    toks = PC.tokens(cfg, 30, 7)
    want = O.forward(cfg, w, toks)
    cache = model.alloc_cache(4, 16, torch.float32, state_slots=2)
    table = [0, 1, 2, 3]
    model.forward(ForwardBatch.build([toks[:20]], [0], [table], 16, state_slots=[1]), cache)
    drafts = toks[20:23] + [t for t in range(5) if t != toks[23]][:2]
    batch = ForwardBatch.build([drafts], [20], [table], 16, state_slots=[1], has_state=[True])
    batch.spec_verify = True
    model.forward(batch, cache)
    model.commit_spec([3], cache)
    got = model.compute_logits(model.forward(ForwardBatch.build([toks[23:]], [23], [table], 16, state_slots=[1], all_logits=True), cache))
    assert PC.spread(got, want[23:]) < TOL


def test_two_tensor_parallel_ranks_reproduce_the_whole_model(folder):
    from atlas_b200.layers import ParallelCtx
    from atlas_b200.parallel.comm import FakeWorld
    path, cfg, w = folder("even")
    toks = PC.tokens(cfg, 40, 8)
    world = FakeWorld(2, timeout_s=60.0)

    def rank(r):
        comm = world.comm(r)
        model = load_model(path, ParallelCtx(tp_rank=r, tp_size=2, comm=comm, ep_comm=comm), dtype="float32", max_pos=64)
        return model.forward_dense_reference(toks)
    want = O.forward(cfg, w, toks)
    for got in world.run(rank):
        assert PC.spread(got, want) < TOL


def test_configuration_reads_every_size():
    cfg, _ = PC.CASES["wide"]
    c = ModelConfig.from_hf(cfg)
    a = c.for_layer(0)
    assert (c.model_type, c.family, c.vocab_size, c.hidden_size, c.residual_streams) == ("papidra", "hybrid", 77, 100, 5)
    assert (a.num_attention_heads, a.num_key_value_heads, a.head_dim, a.v_head_dim, a.attn_cache_width) == (20, 1, 72, 40, 128)
    assert (a.attn_chunk, a.rotary_dim, a.mamba_conv_kernel, a.ssm_state_size, a.mamba_norm_groups) == (33, 36, 5, 136, 1)
    assert (a.glu_limit, a.intermediate_size, c.for_layer(1).wkv_head_dim, c.layer_specs[1].has_mlp) == (1.5, 36, 72, False)
    with pytest.raises(ValueError):
        ModelConfig.from_hf({**cfg, "layers": [{"type": "other", "mixer": {}, "mlp": None}]})


def test_yarn_table_matches_the_plain_frequencies():
    from atlas_b200.config import _rotary_overrides
    from atlas_b200.ops import reference as ref
    for rot in ({"dims": 16, "base": 1e4, "scaling": {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}},
                {"dims": 64, "base": 5e5, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}},
                {"dims": 6, "base": 100.0, "scaling": {"factor": 0.5, "original": 7, "fast": 1.0, "slow": 1.0}},
                {"dims": 2, "base": 1e4, "scaling": None}):
        o = _rotary_overrides(rot)
        table = ref.build_rope_cache(o["rotary_dims"], 50, o["rope_theta"], o["rope_scaling"])
        x = torch.randn(50, 1, rot["dims"] + 4, generator=torch.Generator().manual_seed(0))
        got = ref.apply_rope(x, torch.arange(50), table, rot["dims"])
        assert (got - O.rotate(x.double(), rot, torch.arange(50))).abs().max() < 1e-5


def test_random_preset_serves_through_the_command_line_loader():
    from types import SimpleNamespace
    from atlas_b200.cli import load_for_serving
    from atlas_b200.layers import ParallelCtx
    args = SimpleNamespace(model="preset:tiny-papidra", quantization="auto", dtype=None, max_seq_len=256, seed=0)
    model, _ = load_for_serving(args, ParallelCtx(), torch.device("cpu"))
    eng = LLMEngine(model, EngineConfig(num_kv_blocks=32, max_num_seqs=2, max_seq_len=128, kv_cache_dtype="fp8"))
    out = eng.generate([[1, 2, 3]], SamplingParams(max_tokens=5, ignore_eos=True))
    assert len(out[0].output_tokens) == 5


def test_trace_runner_writes_what_was_asked_for(folder, tmp_path):
    """The command itself: steps on standard input, one file per step with wanted places, an answer after every step."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np
    path, cfg, w = folder("ones")
    toks = PC.tokens(cfg, 12, 4)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:9], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": toks[:4], "want": [3, 0]}, {"id": "x", "tokens": toks[9:], "want": [1]}], "end": ["x"]},
             {"step": 7, "entries": [{"id": "y", "tokens": toks[4:5], "want": [0]}], "end": ["y"]}]
    runner = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    r = subprocess.run([sys.executable, runner, "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128",
                        "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split("\n")[:3] == ["done 0", "done 1", "done 7"] and sorted(os.listdir(tmp_path)) == ["1.f32", "7.f32"]
    want = O.forward(cfg, w, toks)
    got = torch.from_numpy(np.fromfile(tmp_path / "1.f32", dtype="<f4")).view(3, -1)
    assert PC.spread(got, want[[3, 0, 10]]) < TOL
    assert PC.spread(torch.from_numpy(np.fromfile(tmp_path / "7.f32", dtype="<f4")).view(1, -1), want[4:5]) < TOL


@pytest.mark.parametrize("kind", ["wkv", "parallel"])
def test_models_of_one_layer_kind(tmp_path, kind):
    layer = PC.wkv_layer(2, 24, PC.ff(32, 1.0)) if kind == "wkv" else PC.par_layer(PC.attn(2, 2, 16, 16, 20, 8), PC.mamba(2, 16, 16, 2, 1, 4))
    PC.CASES["one kind"] = (PC.model(50, 48, 3, [layer, layer]), 8)
    try:
        cfg, w = PC.write(str(tmp_path), "one kind")
    finally:
        del PC.CASES["one kind"]
    toks = PC.tokens(cfg, 45, 1)
    eng = build_engine(str(tmp_path), "float32", 64, device="cpu")
    assert PC.spread(PC.feed_alone(eng, "a", toks, PC.portions(45, [7, 1, 20])), O.forward(cfg, w, toks)) < TOL
