"""Papidra on the GPU: every kernel of its mechanisms against the plain statement, then whole models through the engine in
bf16 and fp32 (portions, unequal batches, reused pages and slots, decode graphs, generation)."""
import math
from types import SimpleNamespace

import pytest
import torch

import papidra_cases as PC
import papidra_oracle as O

pytestmark = pytest.mark.gpu
DTYPES = [torch.bfloat16, torch.float32]
REL = {torch.bfloat16: 1.2e-2, torch.float32: 2e-5}


def rnd(*shape, seed=0, std=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std


def close(got, want, dtype, what="", factor=1.0):
    got, want = got.detach().cpu().double(), want.double()
    err = (got - want).abs().max().item()
    assert err <= factor * REL[dtype] * max(want.abs().max().item(), 1e-3), f"{what}: {err} of {want.abs().max().item()}"


def rounded(t, dtype):
    return t.to(dtype).double()


def batch_of(lens, live, slots):
    """The part of a ForwardBatch that recurrent layers read."""
    return SimpleNamespace(query_lens_host=list(lens), state_slots_host=list(slots), has_state_host=list(live), snapshot_plan={})


# ------------------------------------------------------------------------------------------------- streams
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,W,T", [(1, 64, 3), (2, 96, 5), (3, 90, 4), (4, 1024, 7), (5, 101, 2), (8, 260, 3), (3, 12288, 2)])
def test_hyper_norm(dtype, S, W, T):
    from atlas_b200 import ops
    dev, eps = "cuda", 1e-5
    x, y, y2 = rnd(T, S, W, seed=1), rnd(T, W, seed=2).to(dtype), rnd(T, W, seed=3).to(dtype)
    read, write, mix = rnd(S, seed=4), rnd(S, seed=5), rnd(S, S, seed=6)
    nw, w1, w2 = rnd(W, seed=7), rnd(W, seed=8), rnd(W, seed=9)
    conn = SimpleNamespace(mix=mix.to(dev), write=write.to(dev))
    to = lambda t: t.to(dev)

    def after(yy):
        return torch.einsum("st,nsw->ntw", mix.double(), x.double()) + write.double()[None, :, None] * yy[:, None, :]

    def check(delta, streams, want, store=True):
        got, s = ops.hyper_norm(streams, delta, to(read), to(nw), eps, write=store)
        u = torch.einsum("s,nsw->nw", read.double(), want)
        close(got, O.rms(u, eps) * nw.double(), dtype, "normed")
        close(s, want if store else x, torch.float32, "streams", factor=10)
    check(ops.StreamDelta(to(y), scale=2.5), None, (y.double() * 2.5)[:, None].expand(T, S, W))
    check(ops.StreamDelta(to(y), conn), to(x), after(y.double()))
    both = 0.5 * (O.rms(y.double(), eps) * w1.double() + O.rms(y2.double(), eps) * w2.double())
    check(ops.StreamDelta(to(y), conn, y2=to(y2), w1=to(w1), w2=to(w2)), to(x), after(both))
    got, s = ops.hyper_norm(to(x), ops.StreamDelta(to(y), conn), to(read), to(nw), eps, write=False)
    assert torch.equal(s.cpu(), x)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [64, 90, 1028])
def test_token_shift(dtype, W):
    from atlas_b200.ops import cuda as K
    lens, live, slots = [1, 19, 2, 1, 9], [True, False, True, False, True], [3, 0, 4, 1, 2]
    x, mu, shift = rnd(sum(lens), W).to(dtype), rnd(5, W, seed=1), rnd(6, W, seed=2).to(dtype)
    got = K.token_shift_mix(x.cuda(), mu.cuda(), batch_of(lens, live, slots), shift.cuda())
    want, t0 = torch.empty(5, sum(lens), W, dtype=torch.float64), 0
    for n, a, s in zip(lens, live, slots):
        first = shift[s:s + 1].double() if a else torch.zeros(1, W).double()
        h = x[t0:t0 + n].double()
        prev = torch.cat([first, h[:-1]])
        want[:, t0:t0 + n] = h + (prev - h) * mu.double()[:, None]
        t0 += n
    close(got, want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [8, 24, 45, 1536])
def test_clamped_glu_meets_its_limits(dtype, n):
    from atlas_b200 import ops
    gu = rnd(6, 2 * n, std=3.0).to(dtype)
    for limit in (0.5, 1.0, 7.0):
        close(ops.gated_unit_act(gu.cuda(), (limit, 1.702, 1.0)).x, O.clamped_glu(gu[:, :n].double(), gu[:, n:].double(), limit), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("groups,size", [(1, 8), (3, 10), (4, 64), (2, 1100), (1, 4096)])
def test_group_norm_gate(dtype, groups, size):
    from atlas_b200 import ops
    n, eps = groups * size, 1e-5
    y, zz, w = rnd(5, n, seed=1).to(dtype), rnd(5, n + 6, seed=2).to(dtype), rnd(n, seed=3)
    for off in (0, 3):
        z = zz[:, off:off + n]
        gate, split = O.silu(z.double()), lambda t: O.rms(t.view(5, groups, size), eps).reshape(5, n) * w.double()
        close(ops.group_norm_gate(y.cuda(), zz.cuda()[:, off:off + n], w.cuda(), size, eps, True), split(y.double() * gate), dtype)
        close(ops.group_norm_gate(y.cuda(), zz.cuda()[:, off:off + n], w.cuda(), size, eps, False), split(y.double()) * gate, dtype)


# ------------------------------------------------------------------------------------------------- recurrences
LENS = [([1, 1, 1], [True, False, True]), ([37, 1, 2, 18], [False, True, True, False]), ([16, 17, 33], [True, True, False])]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("lens,live", LENS, ids=["decode", "mixed", "rows16"])
@pytest.mark.parametrize("H,D", [(1, 8), (3, 16), (2, 40), (2, 64), (1, 72), (1, 130)])
def test_wkv_scan(dtype, lens, live, H, D):
    """State carried in, unequal lengths, a far memory: some channels hardly decay, some forget at once."""
    from atlas_b200.ops import cuda as K
    T, n, W = sum(lens), H * D, 37
    r, k, v, raw = (rnd(T, n, seed=i).to(dtype) for i in range(4))
    w0, u = torch.linspace(-9.0, 1.0, n), rnd(H, D, seed=5)
    x = rnd(T, W, seed=6).to(dtype)
    slots = [4, 1, 0, 2][:len(lens)]
    h0, sh0 = rnd(5, H, D, D, seed=7), rnd(5, W, seed=8).to(dtype)
    layer = SimpleNamespace(w0=w0.cuda(), u=u.cuda(), inner=n, h=H, d=D)
    state = {"h": h0.cuda(), "shift": sh0.cuda()}
    args = [t.cuda() for t in (x, r, k, v, raw)]
    dry = K.wkv_forward(layer, *args, batch_of(lens, live, slots), state, False)
    assert torch.equal(state["h"].cpu(), h0) and torch.equal(state["shift"].cpu(), sh0)
    got = K.wkv_forward(layer, *args, batch_of(lens, live, slots), state, True)
    assert torch.equal(dry, got)
    t0, hs = 0, lambda t: t.double().view(-1, H, D)
    decay = torch.exp(-torch.exp(raw.double() + w0.double())).view(T, H, D)
    keep = set(range(5)) - set(slots)
    for m, a, s in zip(lens, live, slots):
        rows = slice(t0, t0 + m)
        S = h0[s].double().transpose(1, 2) if a else torch.zeros(H, D, D).double()
        for t in range(t0, t0 + m):
            kv = hs(k)[t][:, :, None] * hs(v)[t][:, None, :]
            o = ((S + u.double()[:, :, None] * kv) * hs(r)[t][:, :, None]).sum(1)
            close(got[t].view(H, D), o, dtype, f"row {t - t0}", factor=4)
            S = decay[t][:, :, None] * S + kv
        close(state["h"][s].transpose(1, 2), S, torch.float32, "state", factor=20)
        assert torch.equal(state["shift"][s].cpu(), x[rows][-1])
        t0 += m
    for s in keep:
        assert torch.equal(state["h"][s].cpu(), h0[s])


def test_wkv_from_zero_state_matches_the_plain_recurrence():
    from atlas_b200.ops import cuda as K
    T, H, D = 150, 2, 48
    r, k, v, raw = (rnd(T, H * D, seed=i) for i in range(4))
    w0, u = torch.linspace(-8.0, 0.0, H * D), rnd(H, D, seed=5)
    layer = SimpleNamespace(w0=w0.cuda(), u=u.cuda(), inner=H * D, h=H, d=D)
    state = {"h": torch.full((1, H, D, D), 9.0).cuda(), "shift": torch.zeros(1, 8).cuda()}
    got = K.wkv_forward(layer, rnd(T, 8).cuda(), r.cuda(), k.cuda(), v.cuda(), raw.cuda(), batch_of([T], [False], [0]), state, True)
    z = lambda t: t.double().view(T, H, D)
    want = O.wkv_recurrence(z(r), z(k), z(v), torch.exp(-torch.exp(raw.double() + w0.double())).view(T, H, D), u.double())
    close(got.view(T, H, D), want, torch.float32, factor=5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("lens,live", LENS, ids=["decode", "mixed", "rows16"])
@pytest.mark.parametrize("H,P,N,G,W", [(1, 8, 8, 1, 1), (6, 24, 24, 3, 3), (4, 32, 64, 2, 4), (2, 20, 136, 2, 5), (3, 150, 13, 1, 2)])
def test_mamba2_conv_and_scan(dtype, lens, live, H, P, N, G, W):
    from atlas_b200.ops import cuda as K
    T, inner = sum(lens), H * P
    C = inner + 2 * G * N
    proj = rnd(T, C + H, std=0.7).to(dtype)
    cw, cb = rnd(C, W, seed=1, std=0.5).to(dtype), rnd(C, seed=2).to(dtype)
    A, Dk, db = rnd(H, seed=3), rnd(H, seed=4), rnd(H, seed=5) - 1.0
    slots = [4, 1, 0, 2][:len(lens)]
    h0, c0 = rnd(5, H, P, N, seed=6), rnd(5, C, W - 1, seed=7).to(dtype)
    layer = SimpleNamespace(conv_w=cw.cuda(), conv_b=cb.cuda(), W=W, d_inner=inner, A_log=A.cuda(), D=Dk.cuda(), dt_bias=db.cuda(),
                            cfg=SimpleNamespace(mamba_dt_min=0.0), h=H, p=P, n=N, g=G)
    state = {"h": h0.cuda(), "conv": c0.cuda()}
    pc = proj.cuda()
    got = K.mamba2_forward(layer, pc[:, :C], pc[:, C:], batch_of(lens, live, slots), state, True)
    t0 = 0
    for m, a, s in zip(lens, live, slots):
        x = proj[t0:t0 + m, :C].double()
        past = c0[s].double().T if a else torch.zeros(W - 1, C).double()
        full = torch.cat([past, x])
        conv = O.silu(cb.double() + sum(full[i:i + m] * cw.double()[:, i] for i in range(W)))
        conv = rounded(conv, dtype)
        dt = O.softplus(proj[t0:t0 + m, C:].double() + db.double())
        xs, b, c = conv[:, :inner].view(m, H, P), conv[:, inner:inner + G * N].view(m, G, N), conv[:, inner + G * N:].view(m, G, N)
        S = h0[s].double() if a else torch.zeros(H, P, N).double()
        g = torch.arange(H) // (H // G)
        for t in range(m):
            S = torch.exp(-torch.exp(A.double()) * dt[t])[:, None, None] * S + dt[t][:, None, None] * xs[t][:, :, None] * b[t][g][:, None, :]
            y = (S * c[t][g][:, None, :]).sum(-1) + Dk.double()[:, None] * xs[t]
            close(got[t0 + t].view(H, P), y, dtype, f"row {t}", factor=4)
        close(state["h"][s], S, dtype, "state", factor=4)
        assert torch.equal(state["conv"][s].cpu().double(), full[m:].T if W > 1 else state["conv"][s].cpu().double())
        t0 += m


@pytest.mark.parametrize("kind", ["wkv", "mamba2"])
def test_snapshots_and_row_limits(kind):
    """A snapshot in the middle of a chunk and a fold of the first rows leave exactly the state after those rows."""
    from atlas_b200.ops import cuda as K
    H, D, T, cut = 2, 24, 41, 19
    if kind == "wkv":
        layer = SimpleNamespace(w0=torch.linspace(-6, 0, H * D).cuda(), u=rnd(H, D).cuda(), inner=H * D, h=H, d=D)
        ins = [rnd(T, H * D, seed=i).cuda() for i in range(5)]                       # x, r, k, v, raw
        fresh = lambda: {"h": torch.zeros(4, H, D, D).cuda(), "shift": torch.zeros(4, H * D).cuda()}
        run = lambda n, b, st: K.wkv_forward(layer, *[t[:n] for t in ins], b, st, True)
        fold = lambda st: K.wkv_commit(layer, ins[0], *ins[2:], [T], [0], [False], st, [cut])
    else:
        C = H * D + 2 * 16
        layer = SimpleNamespace(conv_w=rnd(C, 4).cuda(), conv_b=rnd(C).cuda(), W=4, d_inner=H * D, A_log=rnd(H).cuda(), D=rnd(H).cuda(),
                                dt_bias=rnd(H).cuda(), cfg=SimpleNamespace(mamba_dt_min=0.0), h=H, p=D, n=16, g=1)
        xbc, dt = rnd(T, C, seed=1).cuda(), rnd(T, H, seed=2).cuda()
        fresh = lambda: {"h": torch.zeros(4, H, D, 16).cuda(), "conv": torch.zeros(4, C, 3).cuda()}
        run = lambda n, b, st: K.mamba2_forward(layer, xbc[:n], dt[:n], b, st, True)
        fold = lambda st: K.mamba2_commit(layer, xbc, dt, [T], [0], [False], st, [cut])
    want, snap, part = fresh(), fresh(), fresh()
    run(cut, batch_of([cut], [False], [0]), want)
    b = batch_of([T], [False], [0])
    b.snapshot_plan = {0: [(cut, 3)]}
    run(T, b, snap)
    fold(part)
    for n in want:
        assert torch.allclose(snap[n][3], want[n][0], atol=1e-5) and torch.allclose(part[n][0], want[n][0], atol=1e-5)


# ------------------------------------------------------------------------------------------------- attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,size", [(4, 2, 64, 24), (3, 3, 128, 16), (20, 1, 64, 33), (6, 1, 256, 160), (2, 1, 64, 1), (4, 4, 64, 0)])
def test_chunked_attention_with_sinks(dtype, H, G, D, size):
    """Rows of prompts and decode rows over scattered pages.  One key near every edge of a chunk is aligned with all queries,
    so that a key too many or too few changes the output by its whole value; the sink is far from negligible."""
    from atlas_b200 import ops
    from atlas_b200.ops import cuda as K
    bs, dev = 16, "cuda"
    reqs = [(150, 1), (97, 1), (64, 1), (210, 77), (49, 2), (40, 40)]           # (tokens in the cache after the step, new rows)
    nblk = sum((L + bs - 1) // bs for L, _ in reqs)
    perm = torch.randperm(nblk, generator=torch.Generator().manual_seed(3)).tolist()
    kc, vc = K.alloc_kv_cache(nblk, bs, G, D, dtype, dev)
    width = max((L + bs - 1) // bs for L, _ in reqs)
    tables = torch.zeros(len(reqs), width, dtype=torch.int32)
    dirn = torch.nn.functional.normalize(rnd(D, seed=11), dim=0) * math.sqrt(D)
    sinks = rnd(H, seed=12, std=1.0) + 2.0
    scale = D ** -0.5
    qs, ks, vs = [], [], []
    for i, (L, n) in enumerate(reqs):
        k, v, q = rnd(L, G, D, seed=20 + i, std=0.3), rnd(L, G, D, seed=40 + i), rnd(n, H, D, seed=60 + i, std=0.3) + dirn * 0.5
        step = size or 50
        for e in range(0, L, step):
            for p in (e - 1, e, e + 1):
                if 0 <= p < L:
                    k[p] = dirn * 0.6
        blocks = [perm.pop() for _ in range((L + bs - 1) // bs)]
        tables[i, :len(blocks)] = torch.tensor(blocks, dtype=torch.int32)
        qs.append(q.to(dtype)); ks.append(k.to(dtype)); vs.append(v.to(dtype))
        at = torch.arange(L)
        kc[torch.tensor(blocks)[at // bs].cuda(), (at % bs).cuda()] = ks[-1].cuda()
        vc[torch.tensor(blocks)[at // bs].cuda(), (at % bs).cuda()] = vs[-1].cuda()
    lens = [n for _, n in reqs]
    qsl = torch.tensor([0] + lens).cumsum(0).to(torch.int32)
    batch = SimpleNamespace(block_tables=tables.cuda(), seq_lens=torch.tensor([L for L, _ in reqs], dtype=torch.int32).cuda(),
                            query_start_loc=qsl.cuda(), num_decodes=3, num_seqs=len(reqs), query_lens_host=lens,
                            seq_lens_host=[L for L, _ in reqs], max_seq_len=max(L for L, _ in reqs))
    for sk in (sinks, None):
        got = ops.paged_attention(torch.cat(qs).cuda(), kc, vc, batch, scale, chunk=size, sinks=None if sk is None else sk.cuda())
        for i, (L, n) in enumerate(reqs):
            vis = O.chunk_visible(L, size or L)[L - n:]
            for h in range(H):
                s = (qs[i][:, h].double() @ ks[i][:, h // (H // G)].double().T) * scale
                p = O.sink_softmax(s, vis, (sk if sk is not None else torch.full((H,), -1e30))[h].double())
                close(got[qsl[i]:qsl[i + 1], h], p @ vs[i][:, h // (H // G)].double(), dtype, f"request {i} head {h}", factor=2)
    if size:
        # decode split over several CTAs (as with a long context) gives the same rows
        K._FORCE_DECODE_SPLITS, keep = 3, K._FORCE_DECODE_SPLITS
        try:
            again = ops.paged_attention(torch.cat(qs).cuda(), kc, vc, batch, scale, chunk=size, sinks=sinks.cuda())
        finally:
            K._FORCE_DECODE_SPLITS = keep
        one = ops.paged_attention(torch.cat(qs).cuda(), kc, vc, batch, scale, chunk=size, sinks=sinks.cuda())
        close(again, one.cpu(), dtype, factor=1.5)


def test_rope_write_32bit_places_rotated_keys():
    from atlas_b200 import ops
    from atlas_b200.ops import cuda as K
    from atlas_b200.ops import reference as ref
    T, H, G, D, rot = 21, 3, 2, 64, 20
    kc, vc = K.alloc_kv_cache(4, 16, G, D, torch.float32, "cuda")
    q, k, v = rnd(T, H, D), rnd(T, G, D, seed=1), rnd(T, G, D, seed=2)
    table = ref.build_rope_cache(rot, 200, 1e4)
    pos = torch.arange(100, 100 + T, dtype=torch.int32)
    slot = torch.tensor([(37 + i) % 64 if i != 5 else -1 for i in range(T)], dtype=torch.int32)
    got = ops.qk_norm_rope_kv_write(q.cuda(), k.cuda(), v.cuda(), pos.cuda(), table.cuda(), rot, kc, vc, slot.cuda())
    r = {"dims": rot, "base": 1e4, "scaling": None}
    close(got, O.rotate(q.double(), r, pos), torch.float32)
    kr = O.rotate(k.double(), r, pos)
    for i in range(T):
        if slot[i] >= 0:
            close(kc[slot[i] // 16, slot[i] % 16], kr[i], torch.float32)
            close(vc[slot[i] // 16, slot[i] % 16], v[i], torch.float32)
    assert (kc.abs().sum() > 0) and (kc[2, 10].abs().sum() == 0)            # slot 42 belonged to the skipped row


# ------------------------------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    root = tmp_path_factory.mktemp("papidra_gpu")
    made = {}

    def get(name):
        if name not in made:
            path = str(root / name)
            cfg, w = PC.write(path, name)
            toks = {i: PC.tokens(cfg, n, i) for i, n in enumerate((150, 41, 90, 7))}
            made[name] = (path, cfg, toks, {i: O.forward(cfg, w, t) for i, t in toks.items()})
        return made[name]
    return get


# rounding of a whole bf16 model against the exact logits; a wrong key, a lost state or a missing sink is far above it
MODEL_TOL = {"bfloat16": 0.08, "float32": 1e-4}
SHAPES = {"whole": [[1000], [1000], [1000], [1000]], "decode": [[100, 1], [9, 1], [1], [2, 1]], "portions": [[2, 33, 1, 16], [3, 2], [17, 24], [2]]}


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("name", list(PC.CASES))
def test_models_in_portions_and_batches(folder, name, dtype):
    """Each request alone and all together, in one piece, decoded and in small portions, on one engine whose pages and slots
    are used again and again."""
    from atlas_b200.replay import build_engine
    path, cfg, toks, want = folder(name)
    eng = build_engine(path, dtype, 384)
    tol = MODEL_TOL[dtype]
    cut = lambda i, shape: ([SHAPES[shape][i][0]] + [1] * 200 if shape == "decode" else SHAPES[shape][i])
    for shape in SHAPES:
        plans = {}
        for i, t in toks.items():
            c = PC.portions(len(t), cut(i, shape))
            plans[f"r{i}"] = (t, c, i)
            assert PC.spread(PC.feed_alone(eng, f"a{i}", t, c), want[i]) < tol, (shape, i)
        for r, lg in PC.feed_together(eng, plans).items():
            assert PC.spread(lg, want[int(r[1:])]) < tol, (shape, r, "together")
    assert eng.runner.graph_replays > 0 and eng.pool.num_free == eng.pool.num_blocks
    eng.pool.check_invariants()


@pytest.mark.parametrize("graphs", [True, False])
def test_steps_that_read_nothing_back(folder, graphs):
    """Only the last token's logits are asked for, so nothing makes the host wait for the device in between: every step
    still runs on its own tokens, positions and pages."""
    from atlas_b200.replay import build_engine
    path, cfg, toks, want = folder("mixed")
    eng = build_engine(path, "float32", 384, use_cuda_graphs=graphs)
    for _ in range(3):
        for i, t in toks.items():
            cuts = PC.portions(len(t), [2] + [1] * 200)
            at = 0
            for n in cuts:
                last = at + n == len(t)
                got = eng.feed([(f"r{i}", t[at:at + n], [n - 1] if last else [])], [f"r{i}"] if last else [])[0]
                at += n
            assert PC.spread(got, want[i][-1:]) < MODEL_TOL["float32"]


def test_decode_graph_equals_eager_decode(folder):
    from atlas_b200.replay import build_engine
    path, cfg, toks, want = folder("mixed")
    a = build_engine(path, "float32", 384)
    b = build_engine(path, "float32", 384, use_cuda_graphs=False)
    plans = {f"r{i}": (t, PC.portions(len(t), [20] + [1] * 200), 0) for i, t in toks.items()}
    x, y = PC.feed_together(a, plans), PC.feed_together(b, plans)
    assert a.runner.graph_replays > 0 and b.runner.graph_replays == 0
    for r in plans:
        assert (x[r] - y[r]).abs().max() < 1e-4


@pytest.mark.parametrize("options", [{}, {"max_prefill_tokens": 16}, {"num_kv_blocks": 13, "admission_watermark_tokens": 0},
                                     {"ngram_speculative": True, "num_drafts": 3, "mtp_gate": False}], ids=["plain", "portions", "preempt", "spec"])
def test_greedy_generation_through_the_scheduler(folder, options):
    """Engine, scheduler, sampler and the lag-one decode pipeline in fp32: the continuation is the exact model's argmax."""
    from atlas_b200.config import EngineConfig
    from atlas_b200.engine import LLMEngine
    from atlas_b200.loader.load import load_model
    from atlas_b200.sampling import SamplingParams
    path, cfg, toks, _ = folder("mixed")
    _, w = PC.CASES["mixed"][0], PC.weights(PC.CASES["mixed"][0], PC.CASES["mixed"][1])
    prompts = [toks[1], toks[3], toks[2][:60]]
    prompts.append(prompts[0][:35] + PC.tokens(cfg, 6, 99))
    eng = LLMEngine(load_model(path, device="cuda", dtype="float32", max_pos=256),
                    EngineConfig(**{**{"num_kv_blocks": 64, "max_num_seqs": 4, "max_seq_len": 160, "ssm_checkpoint_interval": 16}, **options}))
    sp = SamplingParams(max_tokens=24, temperature=0.0, ignore_eos=True)
    for _ in range(2):
        for p, o in zip(prompts, eng.generate(prompts, sp)):
            full = p + o.output_tokens
            best = O.forward(cfg, w, full)[len(p) - 1:-1]
            top = best.max(-1).values
            picked = best.gather(-1, torch.tensor(o.output_tokens)[:, None])[:, 0]
            assert len(o.output_tokens) == 24 and (top - picked).max() < 1e-4


def test_sampled_serving_preset_runs_in_bf16():
    from atlas_b200.config import EngineConfig, tiny_papidra
    from atlas_b200.engine import LLMEngine
    from atlas_b200.models import build_model
    from atlas_b200.ops import cuda as K
    from atlas_b200.sampling import SamplingParams
    model = build_model(tiny_papidra("bfloat16"), device="cuda").init_random(0)
    eng = LLMEngine(model, EngineConfig(num_kv_blocks=64, max_num_seqs=4, max_seq_len=256, kv_cache_dtype="fp8"))
    outs = eng.generate([[1, 2, 3] * 9, [4, 5]], SamplingParams(max_tokens=30, temperature=0.8, top_p=0.9, seed=1, ignore_eos=True))
    assert all(len(o.output_tokens) == 30 for o in outs) and K.check_status() == 0
