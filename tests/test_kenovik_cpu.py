"""Kenovik on the CPU path (fp32) against the plain statement in ``kenovik_oracle``: configuration, loader, layers, cache and
state manager, batching, prefix cache, speculation, host tier and generation."""
import math

import pytest
import torch

import kenovik_cases as KC
import kenovik_oracle as O
from atlas_b200.config import EngineConfig, ModelConfig
from atlas_b200.engine import LLMEngine
from atlas_b200.loader.load import load_model
from atlas_b200.replay import build_engine
from atlas_b200.sampling import SamplingParams

TOL = 3e-4


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    root = tmp_path_factory.mktemp("kenovik")
    made = {}

    def get(name):
        if name not in made:
            path = str(root / name)
            made[name] = (path,) + KC.write(path, name)
        return made[name]
    return get


@pytest.mark.parametrize("name", list(KC.CASES))
def test_logits_and_every_layer_run_match_the_plain_statement(folder, name):
    path, cfg, w = folder(name)
    toks = KC.tokens(cfg, 70, 1)
    want, layers = O.forward(w, cfg, toks)
    model = load_model(path, dtype="float32", max_pos=128)
    assert len(model.layers) == len(layers)
    model.capture_layers = tuple(range(len(model.layers)))
    got = model.forward_dense_reference(toks)
    for i, (a, b) in enumerate(zip(model.aux_hidden, layers)):
        assert (a - b).abs().max() < TOL * b.abs().max(), f"layer run {i}"
    assert KC.spread(got, want) < TOL


@pytest.mark.parametrize("cuts", [[2], [1], [3, 16, 1, 7], [21], [22, 2], [64]], ids=str)
def test_logits_do_not_depend_on_the_cut(folder, cuts):
    path, cfg, w = folder("mixed")
    toks = KC.tokens(cfg, 75, 2)
    eng = build_engine(path, "float32", 128, device="cpu")
    got = KC.feed_alone(eng, "a", toks, KC.portions(75, cuts))
    assert KC.spread(got, O.forward(w, cfg, toks)[0]) < TOL
    assert eng.pool.num_free == eng.pool.num_blocks and eng.state_pool.num_free == eng.state_pool.num_slots


def test_unequal_batches_on_reused_pages_and_slots(folder):
    path, cfg, w = folder("mixed")
    eng = build_engine(path, "float32", 256, device="cpu")
    plans = {"a": (KC.tokens(cfg, 60, 3), KC.portions(60, [17, 1, 1, 2]), 0), "b": (KC.tokens(cfg, 5, 4), [1] * 5, 0),
             "c": (KC.tokens(cfg, 90, 5), KC.portions(90, [2, 33, 1]), 1), "d": (KC.tokens(cfg, 31, 6), [31], 3)}
    first = KC.feed_together(eng, plans)
    # the second round starts in another order, so every request sits on pages and a slot that others used before
    second = KC.feed_together(eng, {r: plans[r] for r in ("d", "c", "b", "a")})
    for r, (toks, _, _) in plans.items():
        want = O.forward(w, cfg, toks)[0]
        assert KC.spread(first[r], want) < TOL and KC.spread(second[r], want) < TOL
    eng.pool.check_invariants()


def _greedy(cfg, w, p, n):
    p = list(p)
    for _ in range(n):
        p.append(int(O.forward(w, cfg, p)[0][-1].argmax()))
    return p[-n:]


def test_generation_prefix_cache_preemption_and_host_tier(folder):
    """Greedy generation through the scheduler equals the plain statement's greedy continuation: alone, in a batch, from a
    cached prefix (state snapshots), with so few pages that sequences are preempted, swapped to the host, and with drafts."""
    path, cfg, w = folder("even")
    prompts = [KC.tokens(cfg, n, 10 + n) for n in (40, 9, 33)]
    prompts.append(prompts[0][:35] + KC.tokens(cfg, 6, 99))
    want = [_greedy(cfg, w, p, 6) for p in prompts]
    sp = SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True)
    for kw in ({}, {"max_prefill_tokens": 16}, {"num_kv_blocks": 7, "admission_watermark_tokens": 0},
               {"num_kv_blocks": 7, "admission_watermark_tokens": 0, "swap_space_gb": 0.01},
               {"ngram_speculative": True, "num_drafts": 3, "mtp_gate": False}):
        base = {"num_kv_blocks": 64, "max_num_seqs": 4, "max_seq_len": 96, "ssm_checkpoint_interval": 16}
        eng = LLMEngine(load_model(path, dtype="float32", max_pos=128), EngineConfig(**{**base, **kw}))
        for _ in range(2):
            assert [o.output_tokens for o in eng.generate(prompts, sp)] == want, kw
        if not kw:
            assert eng.radix.stats.hit_tokens > 0


def test_rejected_drafts_leave_the_state_alone(folder):
    """A verify step scores drafts without moving the recurrent states of any pass; committing n rows equals having fed n tokens."""
    from atlas_b200.models import ForwardBatch
    path, cfg, w = folder("mixed")
    model = load_model(path, dtype="float32", max_pos=128)
    toks = KC.tokens(cfg, 30, 7)
    want = O.forward(w, cfg, toks)[0]
    cache = model.alloc_cache(4, 16, torch.float32, state_slots=2)
    table = [0, 1, 2, 3]
    model.forward(ForwardBatch.build([toks[:20]], [0], [table], 16, state_slots=[1]), cache)
    drafts = toks[20:23] + [t for t in range(5) if t != toks[23]][:2]
    batch = ForwardBatch.build([drafts], [20], [table], 16, state_slots=[1], has_state=[True])
    batch.spec_verify = True
    model.forward(batch, cache)
    model.commit_spec([3], cache)
    got = model.compute_logits(model.forward(ForwardBatch.build([toks[23:]], [23], [table], 16, state_slots=[1], all_logits=True), cache))
    assert KC.spread(got, want[23:]) < TOL


def test_two_tensor_parallel_ranks_reproduce_the_whole_model(folder):
    from atlas_b200.layers import ParallelCtx
    from atlas_b200.parallel.comm import FakeWorld
    path, cfg, w = folder("even")
    toks = KC.tokens(cfg, 40, 8)
    want = O.forward(w, cfg, toks)[0]
    for ep in (1, 2):
        world = FakeWorld(2, timeout_s=60.0)

        def rank(r):
            comm = world.comm(r)
            p = ParallelCtx(tp_rank=r, tp_size=2, ep_rank=r if ep == 2 else 0, ep_size=ep, comm=comm, ep_comm=comm)
            return load_model(path, p, dtype="float32", max_pos=64).forward_dense_reference(toks)
        for got in world.run(rank):
            assert KC.spread(got, want) < TOL, ep


def test_passes_share_weights_and_own_their_caches(folder):
    path, cfg, _ = folder("mixed")
    model = load_model(path, dtype="float32", max_pos=64)
    assert [l.number for l in model.layers] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4, 5]
    assert [l.step is not None for l in model.layers] == [i in (1, 4, 7) for i in range(12)]
    assert len(model.weight_layers()) == 6
    a, b, c = (model.layers[i] for i in (2, 5, 8))
    assert a.mixer.in_proj is b.mixer.in_proj is c.mixer.in_proj and a.ffn is c.ffn and a.mixer is not b.mixer
    cache = model.alloc_cache(3, 16, torch.float32, state_slots=1)
    assert sorted(cache.kv) == [0, 1, 3, 4, 6, 7, 9, 11] and sorted(cache.states) == [2, 5, 8, 10]
    assert len({t.data_ptr() for kv in cache.kv.values() for t in kv}) == 16
    per_block = sum(t.numel() * t.element_size() for kv in cache.kv.values() for t in kv) // 3
    assert model.kv_bytes_per_block(16, torch.float32) == per_block


def test_configuration_reads_every_size():
    cfg = KC.CASES["wide"]
    c = ModelConfig.from_hf(cfg)
    d, r, s = (c.for_layer(i) for i in range(3))
    assert (c.model_type, c.vocab_size, c.hidden_size, c.num_hidden_layers, c.loop_steps, c.embed_scale) == ("kenovik", 77, 100, 6, 2, 1.5)
    assert c.input_norms and c.tie_word_embeddings and not c.norm_plus_one
    assert [(x.weights_of, x.step) for x in c.layer_specs] == [(-1, 0), (-1, -1), (-1, -1), (0, 1), (1, -1), (2, -1)]
    assert (d.num_attention_heads, d.num_key_value_heads, d.head_dim, d.v_head_dim, d.attn_cache_width, d.rotary_dim) == (20, 1, 72, 130, 256, 0)
    assert (d.qk_norm_rows, d.attn_distance_reach, d.attn_query_temp, d.attn_query_temp_every, d.attention_bias) == (True, 60, 0.4, 16, False)
    assert (d.num_experts, d.num_experts_per_tok, d.moe_intermediate_size, d.glu_limit, d.router_n_group, d.router_topk_group) == (24, 5, 36, 1.2, 6, 2)
    assert (d.shared_expert_intermediate_size, d.shared_glu_limit, d.routed_scaling_factor, d.router_scoring) == (50, 2.0, 1.7, "sigmoid")
    assert (r.rglru_width, r.rglru_blocks, r.rglru_conv_kernel, r.intermediate_size, r.mlp_activation) == (417, 3, 7, 37, "silu_glu")
    assert (s.rotary_dim, s.rope_theta, s.rope_scaling["rope_type"], s.attn_sink_score, s.attention_bias) == (40, 1e4, "linear", 0.0, True)
    assert [c.is_moe_layer(i) for i in range(6)] == [True, False, True] * 2 and s.shared_expert_intermediate_size == 0
    layer = cfg["layers"][1]
    for bad in ({"layers": [{**layer, "type": "other"}]}, {"layers": [{**layer, "mlp": {"kind": "other"}}]}, {"loop": {"start": 2, "stop": 9, "times": 2}},
                {"layers": [KC.rglru(10, 3, 4)], "loop": None}, {"layers": [KC.rglru(10, 2, 4, KC.moe(5, 1, 8, 2, 1))], "loop": None}):
        with pytest.raises(ValueError):
            ModelConfig.from_hf({**cfg, **bad})


@pytest.mark.parametrize("rows,reach", [(32, 240), (32, 256), (8, 37), (2, 2), (9, 60), (64, 4096), (6, 11), (16, 4)])
def test_distance_buckets(rows, reach):
    """The table per distance equals the plain bucket rule, runs from the first row to the last one without a step back, and a
    distance that meets a bucket's border exactly belongs to the bucket that starts there."""
    from atlas_b200.layers.attention import distance_bucket, distance_table
    rel = torch.arange(rows, dtype=torch.float32)[:, None].expand(rows, 3)
    table = distance_table(rel, reach)
    assert table.shape[0] == 3 and table.shape[1] >= reach + 1 and table[0, -1] == rows - 1
    got = table[1].tolist()
    assert all(b >= a for a, b in zip(got, got[1:])) and got[:rows // 2] == list(range(rows // 2))
    if reach > rows // 2:
        assert got == [O.distance_bucket(n, rows, reach) for n in range(reach + 1)]
        assert distance_bucket(10 ** 6, rows, reach) == rows - 1
        half = rows // 2
        for k in range(rows - half):
            edge = half * (reach / half) ** (k / (rows - half))
            if abs(edge - round(edge)) < 1e-9:
                assert distance_bucket(round(edge), rows, reach) == half + k


def test_interleaved_rotation_with_linear_scaling():
    """Rows reordered at load time and turned half by half give pairs turned in place, the rest of a head untouched."""
    from atlas_b200.config import _rotary_overrides
    from atlas_b200.layers import Attention, ParallelCtx
    from atlas_b200.ops import reference as ref
    for dim, rot in ((16, {"dims": 16, "base": 1e4, "scaling": {"factor": 3.0}}), (24, {"dims": 10, "base": 5e5, "scaling": {"factor": 0.5}}),
                     (8, {"dims": 2, "base": 100.0, "scaling": None})):
        c = ModelConfig(hidden_size=4, num_attention_heads=1, num_key_value_heads=1, head_dim=dim, **_rotary_overrides(rot))
        a = Attention(c, 0, ParallelCtx(), "dense")
        x = torch.randn(50, 1, dim, generator=torch.Generator().manual_seed(0))
        move = lambda t: a._half_split(t[:, 0].t().contiguous()).t()[:, None]
        table = ref.build_rope_cache(c.rotary_dim, 50, c.rope_theta, c.rope_scaling)
        got = ref.apply_rope(move(x), torch.arange(50), table, c.rotary_dim)
        assert (got - move(O.rotate_pairs(x.double(), rot, torch.arange(50)))).abs().max() < 1e-5


def test_recurrence_carried_over_cuts():
    from atlas_b200.ops import reference as ref
    T, C = 60, 7
    g = torch.Generator().manual_seed(2)
    u, zr, zi = (torch.randn(T, C, generator=g) * s for s in (1.0, 4.0, 2.0))
    lam = torch.linspace(-9.0, 3.0, C)
    want = O.gated_linear_recurrence(u.double(), O.sigmoid(zr.double()), O.sigmoid(zi.double()), lam.double())
    h, out = torch.zeros(C), []
    for a, b in ((0, 1), (1, 3), (3, 40), (40, 60)):
        out.append(ref.linear_recurrence(*ref.rglru_gates(u[a:b], zr[a:b], zi[a:b], lam), h))
        h = out[-1][-1]
    assert (torch.cat(out) - want).abs().max() < 1e-5 * want.abs().max()


def test_masked_groups_lose_to_negative_scores():
    """Choice scores are negative everywhere; a closed group must not win with zero."""
    from atlas_b200.ops import reference as ref
    z, corr = torch.zeros(1, 6), torch.tensor([-1.0, -3.0, -2.0, -2.1, -4.0, -4.0])
    w, ids = ref.moe_route(z, 3, True, "sigmoid", corr, 3, 2, 2.0)
    assert sorted(ids[0].tolist()) == [0, 2, 3] and torch.allclose(w, torch.full((1, 3), 2.0 / 3.0))


def test_random_presets_serve_through_the_command_line_loader():
    from types import SimpleNamespace
    from atlas_b200.cli import load_for_serving
    from atlas_b200.config import PRESETS
    from atlas_b200.layers import ParallelCtx
    args = SimpleNamespace(model="preset:tiny-kenovik", quantization="auto", dtype=None, max_seq_len=256, seed=0)
    model, _ = load_for_serving(args, ParallelCtx(), torch.device("cpu"))
    eng = LLMEngine(model, EngineConfig(num_kv_blocks=32, max_num_seqs=2, max_seq_len=128, kv_cache_dtype="fp8"))
    out = eng.generate([[1, 2, 3]], SamplingParams(max_tokens=5, ignore_eos=True))
    assert len(out[0].output_tokens) == 5
    assert 15e9 < PRESETS["kenovik-20b"]().param_count() < 25e9


@pytest.mark.parametrize("kind", ["rglru", "attention", "attention_2"])
@pytest.mark.parametrize("loop", [None, (0, 2, 2), (1, 2, 4), (0, 1, 2)], ids=str)
def test_models_of_one_layer_kind(tmp_path, kind, loop):
    layer = {"rglru": KC.rglru(24, 4, 5, KC.moe(4, 2, 32, 2, 1, shared=(12, 0.5))), "attention": KC.sink(2, 2, 16, 16, 4, KC.dense(20)),
             "attention_2": KC.distance(2, 1, 16, 8, 21, KC.moe(2, 2, 16, 1, 1))}[kind]
    KC.CASES["one kind"] = KC.model(50, 48, [layer, layer], loop)
    try:
        cfg, w = KC.write(str(tmp_path), "one kind")
    finally:
        del KC.CASES["one kind"]
    toks = KC.tokens(cfg, 45, 1)
    eng = build_engine(str(tmp_path), "float32", 64, device="cpu")
    assert KC.spread(KC.feed_alone(eng, "a", toks, KC.portions(45, [7, 1, 20])), O.forward(w, cfg, toks)[0]) < TOL


MISTAKES = {"one more": ("attend", lambda f: lambda *a, one_more=False, **k: f(*a, **k)),
            "temperature": ("query_temperature", lambda f: lambda p, t: torch.ones(len(p), dtype=torch.float64)),
            "temperature step": ("query_temperature", lambda f: lambda p, t: f(p - 1, t)),
            "bucket": ("distance_bucket", lambda f: lambda n, *a: f(n + 1, *a)),
            "far bucket": ("distance_bucket", lambda f: lambda n, rows, reach: f(min(n, 30), rows, reach)),
            "step vector": ("layer_runs", lambda f: lambda c: [(i, 0 if t is not None else None) for i, t in f(c)]),
            "tap": ("causal_conv", lambda f: lambda x, w, b: f(x, w.flip(1), b)),
            "decay": ("softplus", lambda f: lambda x: torch.zeros_like(x)),
            "router": ("route", lambda f: lambda h, r, w, p: f(h, {**r, "groups": None}, w, p))}


@pytest.mark.parametrize("mistake", list(MISTAKES))
def test_bounds_reject_plausible_mistakes(folder, monkeypatch, mistake):
    """The plain statement with one thing wrong is far outside the tolerance, so the comparisons above would see it."""
    path, cfg, w = folder("mixed")
    toks = KC.tokens(cfg, 70, 1)
    want = O.forward(w, cfg, toks)[0]
    name, wrong = MISTAKES[mistake]
    monkeypatch.setattr(O, name, wrong(getattr(O, name)))
    assert KC.spread(O.forward(w, cfg, toks)[0], want) > 10 * TOL
    assert math.isfinite(want.abs().max().item())
