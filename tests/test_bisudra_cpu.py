"""Bisudra on the CPU path (fp32) against the plain statement in ``bisudra_oracle``: configuration, loader, layers, cache and state
manager, batching, prefix cache, speculation, host tier and generation."""
import pytest
import torch

import bisudra_cases as BC
import bisudra_oracle as O
from atlas_b200.config import EngineConfig, ModelConfig
from atlas_b200.engine import LLMEngine
from atlas_b200.loader.load import load_model
from atlas_b200.replay import build_engine
from atlas_b200.sampling import SamplingParams

TOL = 3e-4


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    root = tmp_path_factory.mktemp("bisudra")
    made = {}

    def get(name):
        if name not in made:
            path = str(root / name)
            made[name] = (path,) + BC.write(path, name)
        return made[name]
    return get


@pytest.mark.parametrize("name", list(BC.CASES))
def test_logits_and_every_layer_match_the_plain_statement(folder, name):
    path, cfg, w = folder(name)
    toks = BC.tokens(cfg, 70, 1)
    layers = []
    want = O.forward(cfg, w, toks, layers)
    model = load_model(path, dtype="float32", max_pos=128)
    model.capture_layers = tuple(range(len(model.layers)))
    got = model.forward_dense_reference(toks)
    for i, (a, b) in enumerate(zip(model.aux_hidden, layers)):
        assert (a - b).abs().max() < TOL * b.abs().max(), f"layer {i}"
    assert BC.spread(got, want) < TOL


@pytest.mark.parametrize("cuts", [[2], [1], [3, 16, 1, 7], [21], [22, 2], [64]], ids=str)
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_logits_do_not_depend_on_the_cut(folder, name, cuts):
    path, cfg, w = folder(name)
    toks = BC.tokens(cfg, 75, 2)
    eng = build_engine(path, "float32", 128, device="cpu")
    got = BC.feed_alone(eng, "a", toks, BC.portions(75, cuts))
    assert BC.spread(got, O.forward(cfg, w, toks)) < TOL
    assert eng.pool.num_free == eng.pool.num_blocks and eng.state_pool.num_free == eng.state_pool.num_slots


def test_unequal_batches_on_reused_pages_and_slots(folder):
    path, cfg, w = folder("mixed")
    eng = build_engine(path, "float32", 256, device="cpu")
    plans = {"a": (BC.tokens(cfg, 60, 3), BC.portions(60, [17, 1, 1, 2]), 0), "b": (BC.tokens(cfg, 5, 4), [1] * 5, 0),
             "c": (BC.tokens(cfg, 90, 5), BC.portions(90, [2, 33, 1]), 1), "d": (BC.tokens(cfg, 31, 6), [31], 3)}
    first = BC.feed_together(eng, plans)
    # the second round starts in another order, so every request sits on pages and a slot that others used before
    second = BC.feed_together(eng, {r: plans[r] for r in ("d", "c", "b", "a")})
    for r, (toks, _, _) in plans.items():
        want = O.forward(cfg, w, toks)
        assert BC.spread(first[r], want) < TOL and BC.spread(second[r], want) < TOL
    eng.pool.check_invariants()


def test_a_request_may_pause_and_go_on(folder):
    """Steps that leave a request out change neither its pages nor its convolution windows."""
    path, cfg, w = folder("mixed")
    eng = build_engine(path, "float32", 256, device="cpu")
    a, b = BC.tokens(cfg, 40, 21), BC.tokens(cfg, 50, 22)
    got = [eng.feed([("a", a[:11], range(11))])[0]]
    other = [eng.feed([("b", b[i:i + 5], range(5))])[0] for i in range(0, 30, 5)]
    x, y = eng.feed([("b", b[30:31], [0]), ("a", a[11:13], range(2))])
    got, other = got + [y], other + [x]
    other.append(eng.feed([("b", b[31:], range(19))], ["b"])[0])
    got.append(eng.feed([("a", a[13:], range(27))], ["a"])[0])
    assert BC.spread(torch.cat(got), O.forward(cfg, w, a)) < TOL and BC.spread(torch.cat(other), O.forward(cfg, w, b)) < TOL


def _greedy(cfg, w, p, n):
    p = list(p)
    for _ in range(n):
        p.append(int(O.forward(cfg, w, p)[-1].argmax()))
    return p[-n:]


def test_generation_prefix_cache_preemption_and_host_tier(folder):
    """Greedy generation through the scheduler equals the plain statement's greedy continuation: alone, in a batch, from a
    cached prefix (state snapshots), with so few pages that sequences are preempted, swapped to the host, and with drafts."""
    path, cfg, w = folder("mixed")
    prompts = [BC.tokens(cfg, n, 10 + n) for n in (40, 9, 33)]
    prompts.append(prompts[0][:35] + BC.tokens(cfg, 6, 99))
    want = [_greedy(cfg, w, p, 6) for p in prompts]
    sp = SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True)
    for kw in ({}, {"max_prefill_tokens": 16}, {"num_kv_blocks": 7, "admission_watermark_tokens": 0},
               {"num_kv_blocks": 7, "admission_watermark_tokens": 0, "swap_space_gb": 0.01},
               {"ngram_speculative": True, "num_drafts": 3, "mtp_gate": False}, {"self_speculative": True, "num_drafts": 2, "mtp_gate": False}):
        base = {"num_kv_blocks": 64, "max_num_seqs": 4, "max_seq_len": 96, "ssm_checkpoint_interval": 16}
        eng = LLMEngine(load_model(path, dtype="float32", max_pos=128), EngineConfig(**{**base, **kw}))
        for _ in range(2):
            assert [o.output_tokens for o in eng.generate(prompts, sp)] == want, kw
        if not kw:
            assert eng.radix.stats.hit_tokens > 0


def test_host_tier_carries_every_part_of_a_sequence(folder):
    """A block and a state slot that go to the host and come back elsewhere are the same."""
    from atlas_b200.kv.host_tier import HostKVTier
    path, _, _ = folder("mixed")
    cache = load_model(path, dtype="float32", max_pos=64).alloc_cache(4, 16, torch.float32, state_slots=3)
    g = torch.Generator().manual_seed(0)
    for k, v in cache.kv.values():
        k[1] = torch.randn(k[1].shape, generator=g)
        v[1] = torch.randn(v[1].shape, generator=g)
    assert len(cache.states) == len(cache.kv) == 4
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
    """A verify step scores drafts without moving the convolution windows; committing n rows equals having fed n tokens."""
    from atlas_b200.models import ForwardBatch
    path, cfg, w = folder("mixed")
    model = load_model(path, dtype="float32", max_pos=128)
    toks = BC.tokens(cfg, 30, 7)
    want = O.forward(cfg, w, toks)
    for accepted in (3, 1):
        cache = model.alloc_cache(4, 16, torch.float32, state_slots=2)
        table = [0, 1, 2, 3]
        model.forward(ForwardBatch.build([toks[:20]], [0], [table], 16, state_slots=[1]), cache)
        drafts = toks[20:20 + accepted] + [t for t in range(5) if t != toks[20 + accepted]][:2]
        batch = ForwardBatch.build([drafts], [20], [table], 16, state_slots=[1], has_state=[True])
        batch.spec_verify = True
        model.forward(batch, cache)
        model.commit_spec([accepted], cache)
        n = 20 + accepted
        got = model.compute_logits(model.forward(ForwardBatch.build([toks[n:]], [n], [table], 16, state_slots=[1], all_logits=True), cache))
        assert BC.spread(got, want[n:]) < TOL


def test_two_tensor_parallel_ranks_reproduce_the_whole_model(folder):
    from atlas_b200.layers import ParallelCtx
    from atlas_b200.parallel.comm import FakeWorld
    path, cfg, w = folder("even")
    toks = BC.tokens(cfg, 40, 8)
    want = O.forward(cfg, w, toks)
    for ep in (1, 2):
        world = FakeWorld(2, timeout_s=60.0)

        def rank(r):
            comm = world.comm(r)
            p = ParallelCtx(tp_rank=r, tp_size=2, ep_rank=r if ep == 2 else 0, ep_size=ep, comm=comm, ep_comm=comm)
            model = load_model(path, p, dtype="float32", max_pos=64)
            assert model.layers[0].ffn.shard and not model.layers[2].ffn.shard        # whole 128-row shards only
            return model.forward_dense_reference(toks)
        for got in world.run(rank):
            assert BC.spread(got, want) < TOL, ep


def test_one_cached_key_holds_both_maps(folder):
    """A token costs 2 dim + vdim numbers per key / value head (padded): values exist once for the two maps."""
    path, cfg, _ = folder("wide")
    model = load_model(path, dtype="float32", max_pos=64)
    cache = model.alloc_cache(3, 16, torch.float32, state_slots=1)
    assert [tuple(cache.kv[i][0].shape) for i in range(3)] == [(3, 16, 1, 256), (3, 16, 1, 128), (3, 16, 2, 256)]
    assert [model.layers[i].mixer.hq for i in range(3)] == [40, 18, 4]
    per_block = sum(t.numel() * t.element_size() for kv in cache.kv.values() for t in kv) // 3
    assert model.kv_bytes_per_block(16, torch.float32) == per_block


def test_configuration_reads_every_size():
    cfg = BC.CASES["wide"]
    c = ModelConfig.from_hf(cfg)
    a, b, d = (c.for_layer(i) for i in range(3))
    assert (c.model_type, c.vocab_size, c.hidden_size, c.output_norms, c.layer_norms, c.sublayer_gates, c.depth_average) == ("bisudra", 77, 100, True, True, True, True)
    assert (c.input_conv_taps, c.token_side_dim, c.rms_norm_eps, c.tie_word_embeddings) == (2, 13, 1e-5, True)
    assert (a.num_attention_heads, a.num_key_value_heads, a.head_dim, a.v_head_dim, a.attn_cache_width, a.sliding_window) == (20, 1, 70, 130, 256, 33)
    assert (a.rotary_dim, a.rope_theta, a.attn_diff, a.num_experts, a.num_experts_per_tok, a.moe_intermediate_size) == (70, 1e4, 0.3, 20, 5, 36)
    assert (b.attn_cache_width, b.attn_diff, b.intermediate_size, b.mlp_activation, b.num_experts) == (128, 0.4, 50, "relu2", 0)
    assert (d.head_dim, d.v_head_dim, d.attn_cache_width, d.attn_scale) == (128, 256, 256, 128 ** -0.5)
    assert [c.is_moe_layer(i) for i in range(3)] == [True, False, True]
    assert not ModelConfig.from_hf(BC.CASES["mixed"]).layer_specs[2].has_mlp
    one = cfg["layers"][0]
    for bad in ({**one, "type": "other"}, {**one, "mlp": {"kind": "other"}}, {**one, "mlp": BC.moe(3, 4, 8)}, {**one, "mixer": {**one["mixer"], "dim": 129}}):
        with pytest.raises(ValueError):
            ModelConfig.from_hf({**cfg, "layers": [bad]})


def test_random_presets_serve_through_the_command_line_loader():
    from types import SimpleNamespace
    from atlas_b200.cli import load_for_serving
    from atlas_b200.config import PRESETS
    from atlas_b200.layers import ParallelCtx
    args = SimpleNamespace(model="preset:tiny-bisudra", quantization="auto", dtype=None, max_seq_len=256, seed=0)
    model, _ = load_for_serving(args, ParallelCtx(), torch.device("cpu"))
    eng = LLMEngine(model, EngineConfig(num_kv_blocks=32, max_num_seqs=2, max_seq_len=128, kv_cache_dtype="fp8"))
    out = eng.generate([[1, 2, 3]], SamplingParams(max_tokens=5, ignore_eos=True))
    assert len(out[0].output_tokens) == 5
    assert 7e9 < PRESETS["bisudra-8b"]().param_count() < 9e9
    tiny = PRESETS["tiny-bisudra"]()
    held = sum(t.numel() for l in model.layers for t in (l.mixer.in_proj.weight, l.mixer.o.weight, l.gate1.w.weight) + ((l.gate2.w.weight,) if l.gate2 else ()))
    held += sum(l.ffn.experts.w13[:, :144].numel() + l.ffn.experts.w2[..., :72].numel() + l.ffn.router.weight.numel() if l.is_moe else
                l.ffn.gate_up.weight.numel() + l.ffn.down.weight.numel() for l in model.layers if l.ffn is not None)
    assert tiny.param_count() == held + model.embed.numel() + model.side_embed.numel() + 4 * 2 * 20 * 192


@pytest.mark.parametrize("kind", ["dense", "experts", "none"])
def test_models_of_one_layer_kind(tmp_path, kind):
    layer = BC.attention(2, 1, 16, 24, 9, 8, {"dense": BC.ff(40), "experts": BC.moe(3, 2, 32), "none": None}[kind])
    cfg, w = BC.write_model(str(tmp_path), BC.model(50, 48, 3, 6, [layer, layer]))
    toks = BC.tokens(cfg, 45, 1)
    eng = build_engine(str(tmp_path), "float32", 64, device="cpu")
    assert BC.spread(BC.feed_alone(eng, "a", toks, BC.portions(45, [7, 1, 20])), O.forward(cfg, w, toks)) < TOL


@pytest.mark.parametrize("rows", [1, 2, 19])
@pytest.mark.parametrize("map_index", [0, 1])
def test_a_loud_key_at_the_windows_edge(rows, map_index):
    """Just inside the window it takes the weight of its map, just outside it takes none; the other map does not notice."""
    seen = {}
    for back in (36, 37, 0, 5, 48):
        got, want = BC.standing_out("cpu", torch.float32, 4, 2, 20, 24, 37, 12, 70, rows, 69 - back, map_index)
        assert (got - want).abs().max() < 1e-4
        seen[back] = got[-1]
    inside = BC.standing_out("cpu", torch.float32, 4, 2, 20, 24, 0, 12, 70, rows, 32, map_index)[0][-1]
    assert (seen[36] - seen[37])[:, map_index].abs().max() > 0.5 and (inside - seen[37])[:, map_index].abs().max() > 0.5


def test_difference_of_the_maps():
    """With its factor, which the norm behind the output projection hides in a whole model, and a small mean square under eps."""
    from atlas_b200 import ops
    g = torch.Generator().manual_seed(0)
    for dv, D, eps in ((24, 64, 1e-5), (1, 64, 1e-2), (130, 256, 1e-3)):
        a, gate = torch.randn(7, 6, D, generator=g) * 0.1, torch.randn(7, 3 * dv, generator=g)
        want = O.difference(a.double().view(7, 3, 2, D)[..., :dv], 0.45, 0.3, eps).reshape(7, -1)
        assert (ops.map_difference(a, dv, 0.45, 0.7, eps) - want).abs().max() < 1e-5
        assert (ops.map_difference(a, dv, 0.45, 0.7, eps, gate) - want * O.sigmoid(gate.double())).abs().max() < 1e-5


MISTAKES = {
    "window": ("window", lambda f: lambda n, size: f(n, size + 1)),
    "second map left out": ("mix_factor", lambda f: lambda *a: 0.0),
    "constant of the maps": ("mix_factor", lambda f: lambda a, b, c, d, diff: f(a, b, c, d, 0.0)),
    "taps in reverse": ("causal_taps", lambda f: lambda h, w: f(h, w.flip(1))),
    "a tap late": ("causal_taps", lambda f: lambda h, w: torch.cat([torch.zeros_like(h[:1]), f(h, w)[:-1]])),
    "input of the convolution": ("input_convolution", lambda f: lambda h, w: f(h, w) - h),
    "gates open": ("gated", lambda f: lambda y, h, w, name: y),
    "mean left in": ("layer_norm", lambda f: lambda x, w, b, eps: O.unit_rms(x, eps) * w + b),
    "token input": ("token_side", lambda f: lambda x, e, w, pre, eps: x),
    "side embedding": ("token_side", lambda f: lambda x, e, w, pre, eps: f(x, torch.ones_like(e), w, pre, eps)),
    "depth sum": ("depth_average", lambda f: lambda states, factors: states[-1]),
    "depth sum without the embedding": ("depth_average", lambda f: lambda states, factors: f(states[1:], factors[1:])),
    "router bias": ("route", lambda f: lambda h, w, b, top: f(h, w, 0 * b, top)),
    "rotation": ("rotate_pairs", lambda f: lambda x, rot, pos: x),
}


@pytest.mark.parametrize("mistake", list(MISTAKES))
def test_bounds_reject_plausible_mistakes(folder, monkeypatch, mistake):
    """The plain statement with one thing wrong is far outside the tolerance, so the comparisons above would see it."""
    path, cfg, w = folder("mixed")
    toks = BC.tokens(cfg, 70, 1)
    want = O.forward(cfg, w, toks)
    name, wrong = MISTAKES[mistake]
    monkeypatch.setattr(O, name, wrong(getattr(O, name)))
    assert BC.spread(O.forward(cfg, w, toks), want) > 10 * TOL


def test_units_that_a_model_is_compiled_from():
    from atlas_b200 import build
    from atlas_b200.config import tiny_bisudra
    for dtype in ("bfloat16", "float32"):
        units = build.units_for(tiny_bisudra(dtype))
        assert {"differential", "conv1d", "streams", "moe"} <= set(units) and not {"recurrent", "rglru", "mlstm", "latent", "gdn"} & set(units)
