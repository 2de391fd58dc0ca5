"""Tomizen on the CPU path (fp32) against the plain statement in ``tomizen_oracle``: configuration, loader, layers, cache and
state manager, batching, prefix cache, speculation, host tier and generation."""
import pytest
import torch

import tomizen_cases as TC
import tomizen_oracle as O
from atlas_b200.config import EngineConfig, ModelConfig
from atlas_b200.engine import LLMEngine
from atlas_b200.loader.load import load_model
from atlas_b200.replay import build_engine
from atlas_b200.sampling import SamplingParams

TOL = 3e-4


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    root = tmp_path_factory.mktemp("tomizen")
    made = {}

    def get(name):
        if name not in made:
            path = str(root / name)
            made[name] = (path,) + TC.write(path, name)
        return made[name]
    return get


@pytest.mark.parametrize("name", list(TC.CASES))
def test_logits_and_every_layer_match_the_plain_statement(folder, name):
    path, cfg, w = folder(name)
    toks = TC.tokens(cfg, 70, 1)
    layers = []
    want = O.forward(cfg, w, toks, layers)
    model = load_model(path, dtype="float32", max_pos=128)
    model.capture_layers = tuple(range(len(model.layers)))
    got = model.forward_dense_reference(toks)
    for i, (a, b) in enumerate(zip(model.aux_hidden, layers)):
        assert (a - b).abs().max() < TOL * b.abs().max(), f"layer {i}"
    assert TC.spread(got, want) < TOL


@pytest.mark.parametrize("cuts", [[2], [1], [3, 16, 1, 7], [21], [22, 2], [64]], ids=str)
def test_logits_do_not_depend_on_the_cut(folder, cuts):
    path, cfg, w = folder("mixed")
    toks = TC.tokens(cfg, 75, 2)
    eng = build_engine(path, "float32", 128, device="cpu")
    got = TC.feed_alone(eng, "a", toks, TC.portions(75, cuts))
    assert TC.spread(got, O.forward(cfg, w, toks)) < TOL
    assert eng.pool.num_free == eng.pool.num_blocks and eng.state_pool.num_free == eng.state_pool.num_slots


def test_unequal_batches_on_reused_pages_and_slots(folder):
    path, cfg, w = folder("mixed")
    eng = build_engine(path, "float32", 256, device="cpu")
    plans = {"a": (TC.tokens(cfg, 60, 3), TC.portions(60, [17, 1, 1, 2]), 0), "b": (TC.tokens(cfg, 5, 4), [1] * 5, 0),
             "c": (TC.tokens(cfg, 90, 5), TC.portions(90, [2, 33, 1]), 1), "d": (TC.tokens(cfg, 31, 6), [31], 3)}
    first = TC.feed_together(eng, plans)
    # the second round starts in another order, so every request sits on pages and a slot that others used before
    second = TC.feed_together(eng, {r: plans[r] for r in ("d", "c", "b", "a")})
    for r, (toks, _, _) in plans.items():
        want = O.forward(cfg, w, toks)
        assert TC.spread(first[r], want) < TOL and TC.spread(second[r], want) < TOL
    eng.pool.check_invariants()


def _greedy(cfg, w, p, n):
    p = list(p)
    for _ in range(n):
        p.append(int(O.forward(cfg, w, p)[-1].argmax()))
    return p[-n:]


def test_generation_prefix_cache_preemption_and_host_tier(folder):
    """Greedy generation through the scheduler equals the plain statement's greedy continuation: alone, in a batch, from a
    cached prefix (state snapshots), with so few pages that sequences are preempted, swapped to the host, and with drafts."""
    path, cfg, w = folder("mixed")
    prompts = [TC.tokens(cfg, n, 10 + n) for n in (40, 9, 33)]
    prompts.append(prompts[0][:35] + TC.tokens(cfg, 6, 99))
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


def test_host_tier_carries_every_part_of_a_sequence(folder):
    """A block and a state slot that go to the host and come back elsewhere are the same, whatever layer kinds the model has."""
    from atlas_b200.kv.host_tier import HostKVTier
    path, _, _ = folder("mixed")
    cache = load_model(path, dtype="float32", max_pos=64).alloc_cache(4, 16, torch.float32, state_slots=3)
    g = torch.Generator().manual_seed(0)
    for k, v in cache.kv.values():
        k[1] = torch.randn(k[1].shape, generator=g)
        v[1] = torch.randn(v[1].shape, generator=g)
    for st in cache.states.values():
        for t in st.values():
            t[0] = torch.randn(t[0].shape, generator=g)
    tier = HostKVTier(cache, 2, 2)
    slot = tier.alloc_state()
    tier.copy_out([1], [0], 0, slot)
    tier.copy_in([0], [3], slot, 2)
    assert all(torch.equal(t[1], t[3]) for kv in cache.kv.values() for t in kv)
    assert all(torch.equal(t[0], t[2]) for st in cache.states.values() for t in st.values())


def test_rejected_drafts_leave_the_state_alone(folder):
    """A verify step scores drafts without moving the recurrent state; committing n rows equals having fed n tokens."""
    from atlas_b200.models import ForwardBatch
    path, cfg, w = folder("mixed")
    model = load_model(path, dtype="float32", max_pos=128)
    toks = TC.tokens(cfg, 30, 7)
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
    assert TC.spread(got, want[23:]) < TOL


def test_two_tensor_parallel_ranks_reproduce_the_whole_model(folder):
    from atlas_b200.layers import ParallelCtx
    from atlas_b200.parallel.comm import FakeWorld
    path, cfg, w = folder("even")
    toks = TC.tokens(cfg, 40, 8)
    want = O.forward(cfg, w, toks)
    for ep in (1, 2):
        world = FakeWorld(2, timeout_s=60.0)

        def rank(r):
            comm = world.comm(r)
            p = ParallelCtx(tp_rank=r, tp_size=2, ep_rank=r if ep == 2 else 0, ep_size=ep, comm=comm, ep_comm=comm)
            return load_model(path, p, dtype="float32", max_pos=64).forward_dense_reference(toks)
        for got in world.run(rank):
            assert TC.spread(got, want) < TOL, ep


def test_latent_cache_holds_one_row_per_token(folder):
    """The latent layer caches rank + rot numbers per token (padded), not keys and values of every head."""
    path, cfg, _ = folder("mixed")
    model = load_model(path, dtype="float32", max_pos=64)
    cache = model.alloc_cache(3, 16, torch.float32, state_slots=1)
    m = cfg["layers"][1]["mixer"]
    k, v = cache.kv[1]
    assert k.shape == (3, 16, 1, 48 + 16) and v.numel() == 0 and m["kv_rank"] == 40 and m["rot_dim"] == 12
    per_block = sum(t.numel() * t.element_size() for kv in cache.kv.values() for t in kv) // 3
    assert model.kv_bytes_per_block(16, torch.float32) == per_block


def test_configuration_reads_every_size():
    cfg = TC.CASES["wide"]
    c = ModelConfig.from_hf(cfg)
    a, b, m = (c.for_layer(i) for i in range(3))
    assert (c.model_type, c.vocab_size, c.hidden_size, c.output_norms, c.norm_plus_one) == ("tomizen", 77, 100, True, True)
    assert (a.num_attention_heads, a.qk_nope_head_dim, a.qk_rope_head_dim, a.v_head_dim, a.kv_lora_rank, a.sliding_window) == (20, 72, 20, 130, 136, 33)
    assert (a.rotary_dim, a.rope_theta, a.attn_cache_width, a.num_experts, a.num_experts_per_tok, a.moe_intermediate_size) == (20, 1e4, 256, 20, 5, 36)
    assert (b.num_attention_heads, b.num_key_value_heads, b.head_dim, b.v_head_dim, b.attn_cache_width, b.attn_softcap) == (20, 1, 72, 40, 128, 4.0)
    assert b.rotary_dim == 0 and b.qk_norm and not b.qk_norm_plus_one and b.attn_head_gate and not b.norm_topk_prob
    assert (m.mlstm_num_heads, m.mlstm_head_dim, m.mlstm_value_dim, m.mlstm_gate_cap, c.layer_specs[2].has_mlp) == (2, 136, 72, 9.0, False)
    assert [c.is_moe_layer(i) for i in range(3)] == [True, True, False]
    one = {**cfg["layers"][2], "type": "other"}
    with pytest.raises(ValueError):
        ModelConfig.from_hf({**cfg, "layers": [one]})
    with pytest.raises(ValueError):
        ModelConfig.from_hf({**cfg, "layers": [{**cfg["layers"][2], "mlp": {"kind": "dense", "ff": 3}}]})


def test_interleaved_rotation_equals_the_half_split_tables():
    """Rows reordered at load time and turned half by half give the scores of pairs turned in place."""
    from atlas_b200.config import _rotary_overrides
    from atlas_b200.layers.mla import deinterleave_rows
    from atlas_b200.ops import reference as ref
    for rot in ({"dims": 16, "base": 1e4, "scaling": {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}},
                {"dims": 64, "base": 5e5, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}},
                {"dims": 6, "base": 100.0, "scaling": {"factor": 0.5, "original": 7, "fast": 1.0, "slow": 1.0}},
                {"dims": 2, "base": 1e4, "scaling": None}):
        o, n = _rotary_overrides(rot), rot["dims"]
        table = ref.build_rope_cache(o["rotary_dims"], 50, o["rope_theta"], o["rope_scaling"])
        x = torch.randn(50, 1, n, generator=torch.Generator().manual_seed(0))
        got = ref.apply_rope(deinterleave_rows(x[:, 0].t(), n).t()[:, None], torch.arange(50), table, n)
        want = deinterleave_rows(O.rotate_pairs(x.double(), rot, torch.arange(50))[:, 0].t(), n).t()[:, None]
        assert (got - want).abs().max() < 1e-5


def test_gate_recursion_in_log_factors_equals_the_plain_memory():
    """Input gates that jump, forget gates that close: the log factors rebuild S, n and m of the plain recursion, carried on
    from a state that the running maximum has left its start."""
    from atlas_b200.ops import reference as ref
    T, H, D, V, cap = 40, 3, 6, 5, 15.0
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(T, H, n, generator=g) for n in (D, D, V))
    raw, bias = torch.randn(T, 2 * H, generator=g) * 6, torch.randn(2 * H, generator=g)
    i, f = O.log_gates((raw + bias)[:, :H].double(), (raw + bias)[:, H:].double(), cap)
    want, (S, n, m) = O.matrix_memory(q.double(), k.double(), v.double(), i, f)
    h, m0, outs = torch.zeros(H, V + 1, D), torch.zeros(H), []
    for a, b in ((0, 1), (1, 17), (17, 40)):
        la, lb, ms = ref.mlstm_gates(raw[a:b], bias, cap, m0)
        num, dot, h = ref.mlstm_scan(q[a:b], k[a:b], v[a:b], la, lb, h)
        m0 = ms[-1]
        outs.append(num / (torch.maximum(dot.abs(), torch.exp(-ms)) + ref.MLSTM_EPS)[..., None])
    assert (torch.cat(outs) - want).abs().max() < 1e-4 * want.abs().max()
    assert (h[:, :V].transpose(1, 2) - S).abs().max() < 1e-4 and (h[:, V] - n).abs().max() < 1e-4 and (m0 - m).abs().max() < 1e-5


def test_random_presets_serve_through_the_command_line_loader():
    from types import SimpleNamespace
    from atlas_b200.cli import load_for_serving
    from atlas_b200.config import PRESETS
    from atlas_b200.layers import ParallelCtx
    args = SimpleNamespace(model="preset:tiny-tomizen", quantization="auto", dtype=None, max_seq_len=256, seed=0)
    model, _ = load_for_serving(args, ParallelCtx(), torch.device("cpu"))
    eng = LLMEngine(model, EngineConfig(num_kv_blocks=32, max_num_seqs=2, max_seq_len=128, kv_cache_dtype="fp8"))
    out = eng.generate([[1, 2, 3]], SamplingParams(max_tokens=5, ignore_eos=True))
    assert len(out[0].output_tokens) == 5
    assert 12e9 < PRESETS["tomizen-16b"]().param_count() < 20e9


@pytest.mark.parametrize("kind", ["mlstm", "latent_attention", "attention"])
def test_models_of_one_layer_kind(tmp_path, kind):
    layer = {"mlstm": TC.mlstm(2, 24, 12, 4.0, TC.moe(3, 2, 32)), "latent_attention": TC.latent(2, 16, 8, 16, 20, 9),
             "attention": TC.attention(2, 2, 16, 16, 3.0, TC.moe(2, 2, 16))}[kind]
    TC.CASES["one kind"] = TC.model(50, 48, [layer, layer])
    try:
        cfg, w = TC.write(str(tmp_path), "one kind")
    finally:
        del TC.CASES["one kind"]
    toks = TC.tokens(cfg, 45, 1)
    eng = build_engine(str(tmp_path), "float32", 64, device="cpu")
    assert TC.spread(TC.feed_alone(eng, "a", toks, TC.portions(45, [7, 1, 20])), O.forward(cfg, w, toks)) < TOL


@pytest.mark.parametrize("mistake", ["window", "forget gate", "cap", "gate", "expert weights"])
def test_bounds_reject_plausible_mistakes(folder, monkeypatch, mistake):
    """The plain statement with one thing wrong is far outside the tolerance, so the comparisons above would see it.  (The
    memory's denominator is one factor per head, which the norm per head takes out again: it has its own test above.)"""
    path, cfg, w = folder("mixed")
    toks = TC.tokens(cfg, 70, 1)
    want = O.forward(cfg, w, toks)
    if mistake == "window":
        monkeypatch.setattr(O, "window", lambda n, size, f=O.window: f(n, size + 1))
    elif mistake == "forget gate":
        monkeypatch.setattr(O, "log_sigmoid", lambda x: torch.zeros_like(x))
    elif mistake == "cap":
        monkeypatch.setattr(O, "soft_cap", lambda s, cap: s)
    elif mistake == "gate":
        monkeypatch.setattr(O, "sigmoid", lambda x: torch.ones_like(x))
    else:
        monkeypatch.setattr(O, "route", lambda z, top, f=O.route: (f(z, top)[0].sqrt(), f(z, top)[1]))
    assert TC.spread(O.forward(cfg, w, toks), want) > 10 * TOL
