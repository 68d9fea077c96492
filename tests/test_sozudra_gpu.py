"""The kernels and the whole path of the Sozudra design on the GPU, against the plain implementation
(plain_sozudra.py): every mechanism alone, then trace replay under the four schedules in both number formats,
generation through the entry point and its scheduler, and long decoding."""
import io

import pytest
import torch

import plain_sozudra as P
import sozudra_tools as X
import trace_tools as TT
from gpu_tools import paged_setup, rel_err
from model_tools import random_requests

pytestmark = pytest.mark.gpu
F64 = torch.float64
TOL = {torch.float32: 2e-5, torch.bfloat16: 1.6e-2}
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


@pytest.fixture(scope="module")
def K():
    from rvllm_b200.kernels import get_library
    return get_library("cuda:0")


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64) * scale


def dev32(t):
    return t.float().cuda().contiguous()


def ints(*v):
    return torch.tensor(v, dtype=torch.int32).cuda()


# ---------------------------------------------------------------------------------------- stream and embedding
@BOTH
@pytest.mark.parametrize("cols", [44, 45, 320, 1500, 2048, 4096 + 8, 8192, 8192 + 1024])
def test_stream_combine(K, dtype, cols):
    """Every number of terms and norms, on widths on and off the vector path; the norms share one statistic but not their eps."""
    eps = (1e-5, 3e-2)
    x = rnd(5, cols, seed=1).float().double()
    ys = [rnd(5, cols, seed=2 + i, scale=0.7).float().double() for i in range(3)]
    cs = (0.6, -1.25, 0.37)
    gammas = [(rnd(cols, seed=7 + i) + 1.0).to(dtype) for i in range(2)]
    for terms in range(4):
        for norms in range(3):
            got_x = dev32(x)
            same, outs = K.stream_combine(got_x, [(dev32(y), c) for y, c in zip(ys[:terms], cs)],
                                          [(g.cuda(), e) for g, e in zip(gammas[:norms], eps)], dtype)
            want = x + sum(c * y for y, c in zip(ys[:terms], cs)) if terms else x
            assert same is got_x and rel_err(got_x, want) < 1e-6 and len(outs) == norms
            for o, g, e in zip(outs, gammas, eps):
                assert o.dtype == dtype and rel_err(o, P.unit_rms(want, e) * g.double()) < (3e-6 if dtype == torch.float32 else 5e-3)


@BOTH
def test_bigram_rows_in_portions(K, dtype):
    """Portions of one, two and many tokens of three sequences, one of them in no slot: the row of a share's first token
    comes from the state the step before left; products beyond 2^31; a first token after another sequence used the slot."""
    cols, vocab, bigram = 45, 90000, {"buckets": 101, "mul_prev": 65599, "mul_cur": 40503}
    table = rnd(102, cols, seed=3).to(dtype)
    x = rnd(vocab, 1, seed=4).expand(vocab, cols).to(dtype)
    w = {"embed": x.double(), "bigram": table.double()}
    toks = [torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(n)) for n in (31, 12, 4)]
    want = [P.embed(t, w, bigram) for t in toks]
    state = torch.full((3, 1), 77, dtype=torch.int32).cuda()
    slots, done, got = [2, 0, -1], [0, 0, 0], [[], [], []]
    for cut in ((1, 5, 4), (2, 1, 0), (7, 2, 0), (1, 1, 0), (20, 3, 0)):
        live = [s for s in range(3) if cut[s]]
        cu, ids, pos, seq = [0], [], [], []
        for i, s in enumerate(live):
            ids += toks[s][done[s]:done[s] + cut[s]].tolist()
            pos += range(done[s], done[s] + cut[s])
            seq += [i] * cut[s]
            cu.append(len(ids))
        out = K.bigram_add(x[ids].contiguous().cuda(), table.cuda(), ints(*ids), ints(*pos), ints(*seq), ints(*cu), ints(*[slots[s] for s in live]),
                           state, bigram["mul_prev"], bigram["mul_cur"], bigram["buckets"])
        assert out.dtype == torch.float32
        for i, s in enumerate(live):
            got[s].append(out[cu[i]:cu[i + 1]].cpu())
            done[s] += cut[s]
    for s in range(3):
        assert torch.equal(torch.cat(got[s]), want[s].float())
    assert state[:, 0].tolist() == [int(toks[1][-1]), 77, int(toks[0][-1])]


# ---------------------------------------------------------------------------------------- queries, keys, values
def tables(rot, rows=1024):
    from rvllm_b200.parts.rope import RotaryEncoding
    s = rot.get("scaling")
    enc = RotaryEncoding(rot["dims"], rot["base"], None if s is None else dict(s, rope_type="yarn"), rot["dims"])
    enc.prepare(rows, "cuda")
    return enc.rotation_tables()


@BOTH
@pytest.mark.parametrize("maps", [1, 2])
@pytest.mark.parametrize("H,G,D,V,dims,slot", [(6, 2, 24, 16, 16, 48), (4, 4, 8, 12, 4, 16), (3, 3, 9, 14, 6, 32), (8, 2, 64, 64, 64, 128), (2, 1, 128, 256, 128, 256),
                                               (5, 1, 5, 34, 2, 48), (2, 2, 160, 70, 100, 320)])
def test_prepare_queries_keys_values(K, dtype, maps, H, G, D, V, dims, slot):
    """One map with the unit norm and turned values; two maps with biases; what lies beyond a map or a value is zero."""
    T, page, eps = 11, 8, 1e-5
    rot = {"dims": dims, "base": 50.0, "scaling": X.YARN}
    proj = rnd(T, maps * H * D + G * (maps * D + V), seed=10, scale=2.0).float()
    bias = rnd(proj.shape[1], seed=11).float() if maps == 2 else None
    pos = torch.tensor([0, 1, 2, 7, 8, 30, 31, 32, 500, 900, 1023], dtype=torch.int32)
    slots = torch.tensor([5, 6, 7, 16, 17, 40, 41, -1, 3, 2, 1], dtype=torch.int32)
    cache = torch.full((8, 2, G, page, slot), 7.0, dtype=dtype).cuda()
    value_rot = {"dims": V, "base": 50.0} if maps == 1 else None
    q, gate = K.qk_prepare(proj.cuda(), pos.cuda(), *tables(rot), slots.cuda(), cache, H, G, D, V, slot, dtype, eps=eps if maps == 1 else None,
                           halves=True, maps=maps, bias=None if bias is None else bias.cuda(),
                           value_tables=tables(value_rot) if value_rot else None)
    assert gate is None
    x = proj.double() + (bias.double() if bias is not None else 0.0)
    qw, kw = maps * H * D, maps * G * D
    unit = (lambda v: P.unit_rms(v, eps)) if maps == 1 else (lambda v: v)
    want_q = unit(P.turn_halves(x[:, :qw].view(T, H, maps, D), pos, rot))
    want_k = unit(P.turn_halves(x[:, qw:qw + kw].view(T, G, maps, D), pos, rot)).reshape(T, G, maps * D)
    want_v = x[:, qw + kw:].view(T, G, V)
    if value_rot:
        want_v = P.turn_halves(want_v, pos, value_rot)
    tol = 4e-5 if dtype == torch.float32 else 5e-3             # (frequencies are float32: at position 1,023 that shows)
    qv = q.view(T, H, maps, slot).double().cpu()
    for m in range(maps):
        assert rel_err(qv[:, :, m, m * D:(m + 1) * D], want_q[:, :, m]) < tol
        qv[:, :, m, m * D:(m + 1) * D] = 0.0
    assert float(qv.abs().max()) == 0.0
    for t, s in enumerate(slots.tolist()):
        if s < 0:
            continue
        kk, vv = cache[s // page, 0, :, s % page], cache[s // page, 1, :, s % page]
        assert rel_err(kk[:, :maps * D], want_k[t]) < tol and rel_err(vv[:, :V], want_v[t]) < tol
        assert float(kk[:, maps * D:].abs().sum()) == 0.0 and float(vv[:, V:].abs().sum()) == 0.0
    untouched = [s for s in range(8 * page) if s not in set(slots.tolist())]
    assert all(float((cache[s // page, :, :, s % page] - 7.0).abs().max()) == 0.0 for s in untouched)     # slot -1 wrote nothing


@BOTH
@pytest.mark.parametrize("H,V,slot", [(6, 16, 48), (3, 14, 16), (2, 256, 256), (8, 64, 128), (1, 6, 7), (4, 300, 304)])
def test_turn_back_and_map_difference(K, dtype, H, V, slot):
    T, eps = 9, 1e-4
    pos = torch.tensor([0, 1, 2, 7, 31, 32, 100, 640, 1023], dtype=torch.int32)
    o = rnd(T, H, slot, seed=1).to(dtype)
    rot = {"dims": V, "base": 70.0}
    got = K.turn_back(o.view(T, H * slot).cuda(), pos.cuda(), *tables(rot), H, V, slot)
    assert got.dtype == dtype and rel_err(got.view(T, H, V), P.turn_halves(o[..., :V].double(), -pos, rot)) < (4e-5 if dtype == torch.float32 else 5e-3)
    o = rnd(T, H, 2, slot, seed=2).to(dtype)
    o[3] *= 1e-3                                               # a head whose values are of the size of eps
    got = K.map_difference(o.view(T, -1).cuda(), 0.43, eps, 0.7, H, V, slot)
    want = 0.7 * P.unit_rms(o[:, :, 0, :V].double() - 0.43 * o[:, :, 1, :V].double(), eps)
    assert got.dtype == dtype and rel_err(got.view(T, H, V), want) < (2e-6 if dtype == torch.float32 else 5e-3)
    assert rel_err(got.view(T, H, V)[3], want[3]) < (1e-5 if dtype == torch.float32 else 5e-3)


@BOTH
@pytest.mark.parametrize("D,V,page,cap", [(32, 64, 16, None), (12, 20, 8, None), (64, 128, 16, 60.0), (48, 96, 16, None)])
@pytest.mark.parametrize("window", [1, 5, 40, 96, 129, 700])
def test_one_key_of_one_map_at_the_window_edge(K, dtype, D, V, page, cap, window):
    """Two maps on one cached row.  A key whose SECOND map matches the query's second map takes all of that map's weight and
    none of the first's.  Planted at the last position the window still holds it is the result; one position lower it is not
    seen - for a decoded token, the last token of a portion, and both in one step, with the pages below the window given back."""
    H, G, ctx, scale = 2, 1, 900, 40.0 / D ** 0.5
    slot = -(-max(2 * D, V) // 16) * 16
    unit = lambda v: v / torch.sqrt((v * v).mean(-1, keepdim=True))
    wide = lambda v, n: torch.nn.functional.pad(v, (0, n - v.shape[-1]))
    for q_lens, ctxs in (((1,), (ctx,)), ((70,), (ctx,)), ((1, 33), (ctx, 850)), ((2, 1, 1), (ctx, 64, 3))):
        for inside in (True, False):
            k1 = [unit(rnd(c, G, D, seed=50 + i)).to(dtype).double() for i, c in enumerate(ctxs)]
            k2 = [unit(rnd(c, G, D, seed=55 + i)).to(dtype).double() for i, c in enumerate(ctxs)]
            vals = [rnd(c, G, V, seed=60 + i).to(dtype).double() for i, c in enumerate(ctxs)]
            T = sum(q_lens)
            q = unit(rnd(T, H, 2, D, seed=70)).to(dtype)
            at = ctxs[0] - window + (0 if inside else -1)          # the oldest key the first sequence's last query sees, or the one before
            probe = q_lens[0] - 1
            k2[0][at, 0] = unit(q[probe, 1, 1].double()).to(dtype).double()
            rows = torch.zeros(T, H, 2, slot, dtype=dtype)
            rows[:, :, 0, :D], rows[:, :, 1, D:2 * D] = q[:, :, 0], q[:, :, 1]
            keys = [wide(torch.cat([a, b], dim=-1), slot) for a, b in zip(k1, k2)]
            cache, meta = paged_setup(keys, [wide(v, slot) for v in vals], q_lens, page, dtype, seed=window, window=window)
            got = K.paged_attention(rows.view(T, -1).cuda(), cache, meta, 2 * H, G, slot, scale, window, softcap=cap).view(T, H, 2, slot)[..., :V]
            want, t = torch.zeros(T, H, 2, V, dtype=F64), 0
            for a, b, v, n in zip(k1, k2, vals, q_lens):
                c = a.shape[0]
                for i in range(n):
                    p_ = c - n + i
                    lo = max(0, p_ - window + 1)
                    for h in range(H):
                        for m, kk in ((0, a), (1, b)):
                            s = (kk[lo:p_ + 1, 0] @ q[t, h, m].double()) * scale
                            s = s if cap is None else cap * torch.tanh(s / cap)
                            want[t, h, m] = torch.softmax(s, 0) @ v[lo:p_ + 1, 0]
                    t += 1
            assert rel_err(got, want) < (3e-5 if dtype == torch.float32 else 2e-2), (q_lens, inside)
            if cap is None and window > 1:
                assert (rel_err(got[probe, 1, 1], vals[0][at, 0]) < (1e-3 if dtype == torch.float32 else 2e-2)) == inside, (q_lens, inside)
    K.raise_on_abort()


# ---------------------------------------------------------------------------------------- the recurrence
def run_gru(K, w, hs, cuts, slots, width, state, dtype=torch.float32):
    """hs: per sequence [T_s, in]; cuts: per step, per sequence, how many tokens it brings.  Per sequence what the kernel
    gives [T_s, width], the state rows carried from step to step."""
    done, outs = [0] * len(hs), [[] for _ in hs]
    wcat = torch.cat([w["z"], w["x"], w["g"]], dim=0)
    for step in cuts:
        live = [s for s in range(len(hs)) if step[s]]
        parts = [hs[s][done[s]:done[s] + step[s]] for s in live]
        cu = [0]
        for p in parts:
            cu.append(cu[-1] + len(p))
        proj = dev32(torch.cat(parts) @ wcat.T)
        y = K.mingru(proj, dev32(w["z.b"]), dev32(w["x.b"]), ints(*cu), ints(*[slots[s] for s in live]), state, width, cu[-1] == len(live), dtype)
        assert y.dtype == dtype
        for i, s in enumerate(live):
            outs[s].append(y[cu[i]:cu[i + 1]].float().cpu())
            done[s] += step[s]
    return [torch.cat(o) for o in outs]


def gru_weights(width, n_in, seed=0):
    w = {n: rnd(width, n_in, seed=seed + i, scale=0.7).float().double() for i, n in enumerate(("z", "x", "g"))}
    w.update({"z.b": (rnd(width, seed=seed + 5, scale=2.0) - 1.5).float().double(), "x.b": rnd(width, seed=seed + 6).float().double(),
              "o": torch.eye(width, dtype=F64)})
    return w


@BOTH
@pytest.mark.parametrize("width", [1, 33, 96, 130, 512])
def test_min_gru_in_portions_against_the_whole_sequence(K, dtype, width):
    """Portions shorter and longer than a pass of the scan (128 tokens), ending inside and at its edges, beside single
    tokens of other sequences; a sequence in no slot; a slot nobody holds stays as it is."""
    w = gru_weights(width, 12, seed=width)
    hs = [rnd(n, 12, seed=n).float().double() for n in (301, 140, 5)]
    want = [P.min_gru(h, w, "", {"width": width}) for h in hs]
    state = torch.zeros((4, width), dtype=torch.float32, device="cuda")
    state[1].fill_(9.0)
    tol = 3e-6 if dtype == torch.float32 else 5e-3
    got = run_gru(K, w, hs, [(17, 1, 5), (2, 129, 0), (1, 1, 0), (128, 7, 0), (9, 2, 0), (144, 0, 0)], [2, 0, -1], width, state, dtype)
    for a, b in zip(got, want):
        assert rel_err(a, b) < tol
    assert float((state[1] - 9.0).abs().max()) == 0.0 and float(state[3].abs().max()) == 0.0
    left = state[2].clone()
    state.zero_()
    single = run_gru(K, w, hs[:1], [(1,)] * 301, [3], width, state, dtype)
    assert rel_err(single[0], want[0]) < tol and rel_err(state[3], left) < 3e-6


def test_min_gru_keeps_a_value_over_a_long_stretch(K):
    """One token writes with an open gate, every later one with a nearly closed one: a thousand tokens later the state still
    holds that token's candidate - in one portion, and decoded one by one."""
    width, T = 40, 1000
    w = gru_weights(width, 6, seed=3)
    w["z"] = torch.zeros_like(w["z"])
    w["z"][:, 0], w["z.b"] = 40.0, torch.full((width,), -20.0, dtype=F64)
    h = rnd(T, 6, seed=4).float().double()
    h[:, 0] = 0.0
    h[5, 0] = 1.0
    want = P.min_gru(h, w, "", {"width": width})
    u = h[5] @ w["x"].T + w["x.b"]
    c = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    g = h[-1] @ w["g"].T
    assert rel_err(want[-1], c * torch.nn.functional.silu(g)) < 1e-4
    for cuts in ([(T,)], [(3,)] + [(1,)] * (T - 3)):
        state = torch.zeros((1, width), dtype=torch.float32, device="cuda")
        assert rel_err(run_gru(K, w, [h], cuts, [0], width, state)[0], want) < 2e-5


# ---------------------------------------------------------------------------------------- router and experts
@pytest.mark.parametrize("E,top", [(12, 4), (6, 1), (4, 4), (1, 1), (64, 6), (40, 40), (257, 33)])
def test_softmax_router(K, E, top):
    T = 70
    logits, bias = rnd(T, E + 1, seed=E, scale=2.5).float(), rnd(E, seed=top).float()
    chosen, weights, gate = K.moe_route_top(logits.cuda(), bias.cuda(), E, top, 1, 1, 0.0, shared_gate=True, scoring="softmax")
    w = {"router": torch.eye(E, dtype=F64), "router.b": bias.double()}
    want_c, want_w = P.route(logits[:, :E].double(), w, "", {"experts": E, "top": top})
    assert torch.equal(chosen.cpu().sort(-1).values.long(), want_c.sort(-1).values)
    a, b = chosen.cpu().long().argsort(-1), want_c.argsort(-1)
    assert rel_err(weights.cpu().gather(1, a), want_w.gather(1, b)) < 1e-5
    assert rel_err(gate, torch.sigmoid(logits[:, E].double())) < 1e-6


@BOTH
@pytest.mark.parametrize("T,width,ff,E,top", [(1, 48, 24, 5, 2), (9, 44, 9, 4, 4), (70, 384, 88, 12, 3), (300, 64, 40, 3, 1), (260, 192, 96, 12, 4),
                                              (130, 44, 9, 6, 2)])
def test_gated_experts_with_weights_and_a_scaled_addend(K, dtype, T, width, ff, E, top):
    """Few tokens (weights streamed per token) and many (sorted by expert, grouped products): a weight per (token, slot), and a
    factor per token on what is added."""
    x = rnd(T, width, seed=1).to(dtype)
    gu, down = rnd(E, 2 * ff, width, seed=2, scale=width ** -0.5).to(dtype), rnd(E, width, ff, seed=3, scale=ff ** -0.5).to(dtype)
    g = torch.Generator().manual_seed(4)
    chosen = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    weights, factor, add = torch.rand(T, top, generator=g), torch.rand(T, generator=g), rnd(T, width, seed=5).float()
    got = K.moe_experts(x.cuda(), chosen.cuda(), gu.cuda(), down.cuda(), 1.0, add=add.cuda(), out_dtype=torch.float32, weights=weights.cuda(),
                        activation="silu", add_scale=factor.cuda())
    want = add.double() * factor.double()[:, None]
    for e in range(E):
        t, j = torch.nonzero(chosen == e, as_tuple=True)
        w = {"gate": gu[e, :ff].double(), "up": gu[e, ff:].double(), "down": down[e].double()}
        if len(t):
            want[t] += weights[t, j].double()[:, None] * P.gated_expert(x[t].double(), w, "")
    assert got.dtype == torch.float32 and rel_err(got, want) < TOL[dtype]
    K.raise_on_abort()


# ---------------------------------------------------------------------------------------- whole models
LENGTHS = {"a": (45, 170, 33, 81, 1, 138), "b": (90, 37, 300, 64, 151, 2)}
SCHEDULES = {"whole": TT.schedule_whole, "bulk_tail": TT.schedule_bulk_tail, "portions": TT.schedule_portions,
             "mixed": TT.schedule_mixed}
_cache = {}


def _reference(which):
    if which not in _cache:
        from rvllm_b200 import load_config
        folder = X.write_folder({"a": X.small_a, "b": X.small_b}[which](), seed=5, edit=X.lively)
        vocab = load_config(folder).vocab_size
        reqs = random_requests(vocab, LENGTHS[which], seed=4)
        _cache[which] = (folder, vocab, reqs, X.plain_logits(folder, reqs), X.plain_logits(folder, reqs, rounded=True))
    return _cache[which][:4]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("schedule", list(SCHEDULES))
@pytest.mark.parametrize("which", ["a", "b"])
def test_replay_matches_plain(tmp_path, which, schedule, dtype):
    from rvllm_b200.engine import trace as trace_mod
    folder, vocab, reqs, ref = _reference(which)
    trace = SCHEDULES[schedule](reqs)
    block = 8 if which == "a" else 16
    if schedule == "whole":                      # once per configuration as a user runs it: a process of its own
        TT.run_trace_tool(folder, dtype, trace, str(tmp_path), block)
    else:
        engine = trace_mod.build_engine(folder, dtype, trace.max_tokens, block, graphs=schedule == "bulk_tail")
        trace_mod.replay(engine, io.StringIO(trace.lines()), str(tmp_path), io.StringIO())
        engine.cache.check()
        assert not engine.cache.requests
    got = TT.read_logits(str(tmp_path), trace, vocab)
    what = f"{which}/{schedule}/{dtype}"
    if dtype == "float32":
        TT.compare(got, ref, 1e-4, what)
    else:
        TT.compare_bfloat16(got, ref, _cache[which][4], what)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_odd_shapes_whole_and_mixed(tmp_path, dtype):
    """Sizes off every fast path (see sozudra_tools.odd_shapes), whole prompts and the mixed schedule."""
    from rvllm_b200 import load_config
    from rvllm_b200.engine import trace as trace_mod
    folder = X.write_folder(X.odd_shapes(), seed=8, edit=X.lively)
    vocab = load_config(folder).vocab_size
    reqs = random_requests(vocab, (70, 150, 9, 33, 130), seed=6)
    ref = X.plain_logits(folder, reqs)
    rounded = X.plain_logits(folder, reqs, rounded=True) if dtype == "bfloat16" else None
    for name, make in (("whole", TT.schedule_whole), ("mixed", TT.schedule_mixed)):
        out = tmp_path / name
        trace = make(reqs)
        engine = trace_mod.build_engine(folder, dtype, trace.max_tokens, 16)
        trace_mod.replay(engine, io.StringIO(trace.lines()), str(out), io.StringIO())
        engine.cache.check()
        got = TT.read_logits(str(out), trace, vocab)
        if dtype == "float32":
            TT.compare(got, ref, 1e-4, f"odd/{name}")
        else:
            TT.compare_bfloat16(got, ref, rounded, f"odd/{name}")
        del engine


def test_generation_through_the_entry_point():
    """Greedy tokens through LLM.generate and its scheduler (decode steps from CUDA graphs, whose tokens the host has not read
    when the next step is launched; prompts in portions, more requests than slots): float32 equals the plain implementation
    token for token; bfloat16 may differ only where the plain logits' two best lie closer together than its rounding."""
    from rvllm_b200 import LLM, SamplingParams
    folder, vocab, reqs, ref = _reference("b")
    cfg, w = X.read_folder(folder)
    prompts = [reqs["r1"], reqs["r5"], reqs["r3"], reqs["r0"][:50], reqs["r4"][:100]]
    for dtype in ("float32", "bfloat16"):
        llm = LLM(folder, dtype=dtype, block_size=16, num_blocks=40, max_model_len=256, max_num_seqs=3,
                  max_num_batched_tokens=48, max_prefill_chunk=33)
        assert llm.engine.model.graph_safe
        outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=20, ignore_eos=True))
        assert llm.engine.runner._graphs, "decode steps were not replayed from graphs"
        for p, o in zip(prompts, outs):
            got = o.outputs[0].token_ids
            if dtype == "float32":
                assert got == P.greedy(cfg, w, p, 20)
            else:
                ids = list(p)
                for tok in got:
                    logits = P.forward(cfg, w, ids)[-1]
                    top = torch.topk(logits, 2).values
                    assert float(top[0] - top[1]) / float(logits.abs().max()) <= 6e-2 or tok == int(logits.argmax())
                    ids.append(tok)
        assert not llm.engine.cache.requests
        del llm


def test_long_decoding_past_every_window():
    """A short prompt, then 400 tokens one by one (graphs): windows pass over decoded tokens, window pages come back, the
    recurrences run on; the logits equal those of the whole sequence."""
    from rvllm_b200.engine import trace as trace_mod
    from rvllm_b200.engine.step import StepEntry
    folder, vocab, reqs, ref = _reference("a")
    toks = random_requests(vocab, (420,), seed=9)["r0"]
    want = X.plain_logits(folder, {"x": toks})["x"]
    engine = trace_mod.build_engine(folder, "float32", 512, 8, graphs=True)
    engine.runner.step([StepEntry("x", toks[:20], [])])
    for i in range(20, 420):
        logits = engine.runner.step([StepEntry("x", toks[i:i + 1], [0])])
        if i % 57 == 0 or i == 419:
            assert rel_err(logits[0], want[i]) < 1e-4, i
    assert engine.runner._graphs
