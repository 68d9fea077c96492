"""The kernels and the whole path of the Lefolorn design on the GPU, against the plain implementation (plain_lefolorn.py):
every mechanism alone, then trace replay under the four schedules in both number formats, generation through the entry point
and its scheduler, and long decoding."""
import io

import pytest
import torch

import lefolorn_tools as X
import plain_lefolorn as P
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


# ---------------------------------------------------------------------------------------- stream and norms
@BOTH
@pytest.mark.parametrize("cols,groups", [(44, 11), (45, 1), (45, 9), (512, 4), (384, 3), (1536, 4), (1536, 512), (2048, 8), (4096, 4), (4096, 1), (8192, 2),
                                         (8192 + 1024, 9)])
def test_gated_combine(K, dtype, cols, groups):
    """None, one and two terms, with and without a norm, on widths and groups on and off the vector path; a group of another size
    than its neighbours shows in its own columns only."""
    eps = 3e-3
    x = rnd(5, cols, seed=1).float().double()
    x[:, :cols // groups] *= 20.0
    ys = [rnd(5, cols, seed=2 + i, scale=0.7).float().double() for i in range(2)]
    ss = [rnd(cols, seed=4 + i).float().double() for i in range(2)]
    bias, gamma = rnd(2 * cols, seed=6).float().double(), (rnd(cols, seed=7) + 1.0).to(dtype)
    for terms in range(3):
        gates = rnd(5, terms * cols, seed=8, scale=2.0).to(dtype) if terms else None
        want = x.clone()
        for i in range(terms):
            span = slice(i * cols, (i + 1) * cols)
            want += ys[i] * ss[i] * torch.sigmoid(gates[:, span].double() + bias[span])
        for norm in (None, (gamma.cuda(), eps, groups)):
            got_x = dev32(x)
            same, out = K.gated_combine(got_x, [dev32(y) for y in ys[:terms]], [dev32(s) for s in ss[:terms]], gates.cuda() if terms else None,
                                        dev32(bias[:terms * cols]) if terms else None, norm, dtype)
            assert same is got_x and rel_err(got_x, want) < 1e-6 and (out is None) == (norm is None)
            if norm is not None:
                ref = P.grouped_norm(want, gamma.double(), groups, eps)
                assert out.dtype == dtype and rel_err(out, ref) < (3e-6 if dtype == torch.float32 else 5e-3)
    alone = K.grouped_rmsnorm(dev32(x), gamma.cuda(), eps, groups, out_dtype=dtype)
    assert rel_err(alone, P.grouped_norm(x, gamma.double(), groups, eps)) < (3e-6 if dtype == torch.float32 else 5e-3)


# ---------------------------------------------------------------------------------------- queries, keys, values
def tables(rot, rows=1024):
    from rvllm_b200.parts.rope import RotaryEncoding
    enc = RotaryEncoding(rot["dims"], rot["base"], None, rot["dims"])
    enc.prepare(rows, "cuda")
    return enc.rotation_tables()


@BOTH
@pytest.mark.parametrize("H,G,D,V,dims,slot", [(6, 2, 24, 16, 16, 32), (4, 4, 8, 12, None, 16), (3, 3, 9, 14, 6, 16), (8, 2, 64, 64, 64, 64), (2, 1, 128, 256, None, 256),
                                               (5, 1, 5, 34, 2, 48), (2, 2, 300, 70, 100, 304)])
def test_prepare_normed_queries_keys_and_mixed_values(K, dtype, H, G, D, V, dims, slot):
    """Weighted norms in front of the rotation (which would show behind it), biases, temperatures, values that are kept and that
    take a share; what lies beyond a head's elements is zero, a token in no slot writes no key and no value but keeps its value."""
    T, page, eps, lam = 11, 8, 1e-3, 0.37
    rot = {"dims": dims, "base": 50.0}
    extra = 13                                               # columns behind those of q, k and v
    n = H * D + G * (D + V)
    proj = rnd(T, n + extra, seed=10, scale=2.0).float()
    bias, qg, kg, first = rnd(n, seed=11).float(), rnd(D, seed=12).float(), rnd(D, seed=13).float(), rnd(T, G * V, seed=14).float()
    pos = torch.tensor([0, 1, 2, 7, 8, 30, 31, 32, 500, 900, 1023], dtype=torch.int32)
    slots = torch.tensor([5, 6, 7, 16, 17, 40, 41, -1, 3, 2, 1], dtype=torch.int32)
    cs = tables(rot) if dims else (None, None)
    for temp, mode in ((None, "keep"), ((0.6, 8), "mix"), ((-0.1, 1), None)):
        cache = torch.full((8, 2, G, page, slot), 7.0, dtype=dtype).cuda()
        kept = torch.zeros(T, G * V).cuda() if mode == "keep" else None
        q, gate = K.qk_prepare(proj.cuda()[:, :n], pos.cuda(), *cs, slots.cuda(), cache, H, G, D, V, slot, dtype, eps=eps, bias=bias.cuda(),
                               norms=(qg.cuda(), kg.cuda()), temperature=temp, keep_values=kept, mix_values=(first.cuda(), lam) if mode == "mix" else None)
        assert gate is None
        x = proj[:, :n].double() + bias.double()
        turn = (lambda v: P.turn_neighbours(v, pos, rot)) if dims else (lambda v: v)
        want_q = turn(P.unit_rms(x[:, :H * D].view(T, H, D), eps) * qg.double())
        want_q = want_q * P.query_temperature(pos, None if temp is None else {"coef": temp[0], "every": temp[1]})[:, None, None]
        want_k = turn(P.unit_rms(x[:, H * D:H * D + G * D].reshape(T, G, D), eps) * kg.double())
        want_v = x[:, H * D + G * D:].reshape(T, G, V)
        if mode == "keep":
            assert rel_err(kept, want_v.reshape(T, G * V)) < 1e-6
        if mode == "mix":
            want_v = P.mix_values(want_v, {"vmix": torch.tensor(lam, dtype=F64)}, "", {"v_mix": True}, {"first": first.double()})
        tol = 4e-5 if dtype == torch.float32 else 5e-3             # (frequencies are float32: at position 1,023 that shows)
        qv = q.view(T, H, slot).double().cpu()
        assert rel_err(qv[..., :D], want_q) < tol and float(qv[..., D:].abs().sum()) == 0.0
        for t, s in enumerate(slots.tolist()):
            if s < 0:
                continue
            kk, vv = cache[s // page, 0, :, s % page], cache[s // page, 1, :, s % page]
            assert rel_err(kk[:, :D], want_k[t]) < tol and rel_err(vv[:, :V], want_v[t]) < tol
            assert float(kk[:, D:].abs().sum()) == 0.0 and float(vv[:, V:].abs().sum()) == 0.0
        untouched = [s for s in range(8 * page) if s not in set(slots.tolist())]
        assert all(float((cache[s // page, :, :, s % page] - 7.0).abs().max()) == 0.0 for s in untouched)     # slot -1 wrote nothing


@BOTH
@pytest.mark.parametrize("H,V,slot,col0", [(6, 16, 48, 0), (3, 14, 16, 5), (2, 256, 256, 64), (8, 64, 64, 12), (1, 7, 16, 1), (4, 300, 304, 8)])
def test_gate_elements(K, dtype, H, V, slot, col0):
    T = 9
    o, proj = rnd(T, H, slot, seed=1).to(dtype), rnd(T, col0 + H * V + 4, seed=2, scale=3.0).float()
    got = K.gate_elements(o.view(T, H * slot).cuda(), proj.cuda(), col0, H, V, slot)
    want = o[..., :V].double().reshape(T, -1) * torch.sigmoid(proj[:, col0:col0 + H * V].double())
    assert got.dtype == dtype and rel_err(got, want) < (2e-6 if dtype == torch.float32 else 5e-3)


# ---------------------------------------------------------------------------------------- attention with a distance bias
def plain_attention(q, keys, vals, q_lens, scale, **kw):
    """q [T, H, D]; keys, vals per sequence [ctx, G, D]; `table` [rows, H]."""
    H, G, T = q.shape[1], keys[0].shape[1], q.shape[0]
    table, sinks = kw.pop("table", None), kw.pop("sinks", None)
    want, t0 = torch.zeros(T, H, vals[0].shape[2], dtype=F64), 0
    for k, v, n in zip(keys, vals, q_lens):
        c = k.shape[0]
        pos = torch.arange(c)
        for h in range(H):
            full = torch.zeros(c, q.shape[2], dtype=F64)
            full[c - n:] = q[t0:t0 + n, h].double()
            w = P.head_weights(full, k[:, h // (H // G)], pos, scale, table=None if table is None else table[:, h],
                               sink=None if sinks is None else float(sinks[h]), **kw)
            want[t0:t0 + n, h] = (w @ v[:, h // (H // G)])[c - n:]
        t0 += n
    return want


@BOTH
@pytest.mark.parametrize("H,G,D,page", [(8, 2, 64, 16), (6, 2, 32, 8), (4, 1, 128, 16), (3, 3, 48, 16), (28, 4, 128, 64), (5, 1, 16, 16)])
@pytest.mark.parametrize("rows,limit", [(32, 250.0), (6, 9.0), (2, 2.0)])
def test_distance_bias(K, dtype, H, G, D, page, rows, limit):
    """Every distance of prompts, portions and decoded tokens, alone and in one step; tables much shorter and longer than a tile
    of 64 keys, with one added to the denominator."""
    from rvllm_b200.parts.distance import distance_table
    scale = 0.8 / D ** 0.5
    table = rnd(rows, H, seed=rows, scale=1.5).to(dtype)
    bias = distance_table(table.cuda(), limit, G)
    sinks = torch.zeros(H)
    for q_lens, ctxs in (((1,), (700,)), ((331,), (331,)), ((70,), (500,)), ((1, 40, 1, 2), (300, 40, 5, 130)), ((17, 20), (17, 333))):
        keys = [rnd(c, G, D, seed=50 + i).to(dtype).double() for i, c in enumerate(ctxs)]
        vals = [rnd(c, G, D, seed=60 + i).to(dtype).double() for i, c in enumerate(ctxs)]
        q = rnd(sum(q_lens), H, D, seed=70).to(dtype)
        cache, meta = paged_setup(keys, vals, q_lens, page, dtype, seed=rows)
        got = K.paged_attention(q.view(len(q), -1).cuda(), cache, meta, H, G, D, scale, None, sinks=sinks.cuda(), distance_bias=bias)
        want = plain_attention(q, keys, vals, q_lens, scale, table=table.double(), limit=limit, sinks=sinks)
        assert rel_err(got.view(-1, H, D), want) < (3e-5 if dtype == torch.float32 else 2e-2), q_lens
    K.raise_on_abort()


@BOTH
@pytest.mark.parametrize("D,page", [(64, 16), (32, 8), (128, 16), (80, 16)])
@pytest.mark.parametrize("rows,limit", [(32, 250.0), (8, 40.0), (3, 500.0)])
def test_one_far_key_at_a_buckets_edge(K, dtype, D, page, rows, limit):
    """The bias of ONE row of the table is large and every other hugely negative: the result is the mean of the values at exactly
    that row's distances.  For each row, the nearest and the farthest of its distances; with a cap and a window at once."""
    from rvllm_b200.parts.distance import bucket_rows, distance_table
    H, G, ctx = 2, 1, 600
    which = bucket_rows(rows, limit)
    for row in sorted({0, 1, rows // 2 - 1, rows // 2, rows - 2, rows - 1} & set(which)):
        table = torch.full((rows, H), -40.0)
        table[row] = 20.0
        bias = distance_table(table.to(dtype).cuda(), limit, G)
        far = [n for n in range(ctx) if which[min(n, len(which) - 1)] == row]
        for q_lens, window, cap in (((1,), None, None), ((45,), None, None), ((1, 30), None, 3.0), ((40,), far[-1] + 1, None), ((1,), far[-1], 2.0)):
            ctxs = (ctx,) + (77,) * (len(q_lens) - 1)
            keys = [rnd(c, G, D, seed=50 + i, scale=0.3).to(dtype).double() for i, c in enumerate(ctxs)]
            vals = [rnd(c, G, D, seed=60 + i).to(dtype).double() for i, c in enumerate(ctxs)]
            q = rnd(sum(q_lens), H, D, seed=70, scale=0.3).to(dtype)
            if window == 0:
                continue
            cache, meta = paged_setup(keys, vals, q_lens, page, dtype, seed=row, window=window)
            got = K.paged_attention(q.view(len(q), -1).cuda(), cache, meta, H, G, D, 0.01, window, softcap=cap, distance_bias=bias).view(-1, H, D)
            want = plain_attention(q, keys, vals, q_lens, 0.01, table=table.to(dtype).double(), limit=limit, window=window, cap=cap)
            assert rel_err(got, want) < (3e-5 if dtype == torch.float32 else 2e-2), (row, q_lens, window)
            if window is None or window > far[-1]:
                own = vals[0][[ctx - 1 - n for n in far], 0].mean(0)
                assert rel_err(got[q_lens[0] - 1, 0], own) < (2e-2 if dtype == torch.float32 else 5e-2), (row, q_lens)
    K.raise_on_abort()


@BOTH
@pytest.mark.parametrize("D,V,page,cap", [(64, 64, 16, 60.0), (112, 64, 16, None), (12, 20, 8, 50.0)])
@pytest.mark.parametrize("window", [1, 5, 40, 129, 700])
def test_one_key_at_the_window_edge(K, dtype, D, V, page, cap, window):
    """A key that matches a head's query, planted at the last position the window still holds, is the result; one position lower
    it is not seen - for a decoded token, the last token of a portion, and both in one step, pages below the window given back."""
    H, G, ctx, slot = 4, 2, 900, -(-max(D, V) // 16) * 16
    unit = lambda v: v / torch.sqrt((v * v).mean(-1, keepdim=True))
    wide = lambda v: torch.nn.functional.pad(v, (0, slot - v.shape[-1]))
    scale = 40.0 / D
    for q_lens, ctxs in (((1,), (ctx,)), ((70,), (ctx,)), ((1, 33), (ctx, 850)), ((2, 1, 1), (ctx, 64, 3))):
        for inside in (True, False):
            keys = [unit(rnd(c, G, D, seed=50 + i)).to(dtype).double() for i, c in enumerate(ctxs)]
            vals = [rnd(c, G, V, seed=60 + i).to(dtype).double() for i, c in enumerate(ctxs)]
            q = unit(rnd(sum(q_lens), H, D, seed=70)).to(dtype)
            at, probe = ctxs[0] - window + (0 if inside else -1), q_lens[0] - 1
            keys[0][at, 1] = q[probe, 3].double()
            cache, meta = paged_setup([wide(k) for k in keys], [wide(v) for v in vals], q_lens, page, dtype, seed=window, window=window)
            got = K.paged_attention(wide(q).reshape(len(q), -1).cuda(), cache, meta, H, G, slot, scale, window, softcap=cap).view(-1, H, slot)[..., :V]
            want = plain_attention(q, keys, vals, q_lens, scale, cap=cap, window=window)
            assert rel_err(got, want) < (3e-5 if dtype == torch.float32 else 2e-2), (q_lens, inside)
            if window > 1:
                assert (rel_err(got[probe, 3], vals[0][at, 1]) < 3e-2) == inside, (q_lens, inside)
    K.raise_on_abort()


# ---------------------------------------------------------------------------------------- latent attention
@BOTH
@pytest.mark.parametrize("H,D,R,Rq,Kv,gates", [(5, 14, 6, 18, 22, 0), (3, 3, 2, 7, 9, 3), (4, 32, 32, 40, 96, 0), (16, 128, 64, 384, 192, 0), (2, 8, 10, 1, 300, 2)])
def test_latent_rows_and_queries(K, dtype, H, D, R, Rq, Kv, gates):
    T, page, eps = 9, 8, 1e-3
    rot = {"dims": R, "base": 30.0}
    proj = rnd(T, Rq + Kv + R + gates, seed=1, scale=2.0).float()
    qg, cg = (rnd(Rq, seed=2) + 1.0).to(dtype), (rnd(Kv, seed=3) + 1.0).to(dtype)
    pos = torch.tensor([0, 1, 2, 7, 31, 32, 100, 640, 1023], dtype=torch.int32)
    slots = torch.tensor([5, 6, 7, -1, 17, 40, 41, 8, 3], dtype=torch.int32)
    cache = torch.full((8, 1, 1, page, Kv + R), 7.0, dtype=dtype).cuda()
    low, gate = K.latent_down(proj.cuda(), qg.cuda(), cg.cuda(), eps, pos.cuda(), *tables(rot), slots.cuda(), cache, Rq, R, Kv, dtype, heads=gates)
    x, tol = proj.double(), 4e-5 if dtype == torch.float32 else 5e-3
    assert low.dtype == dtype and rel_err(low, P.unit_rms(x[:, :Rq], eps) * qg.double()) < tol
    line = torch.cat([P.unit_rms(x[:, Rq:Rq + Kv], eps) * cg.double(), P.turn_neighbours(x[:, Rq + Kv:Rq + Kv + R], pos, rot)], dim=1)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert rel_err(cache[s // page, 0, 0, s % page], line[t]) < tol
    assert all(float((cache[s // page, 0, 0, s % page] - 7.0).abs().max()) == 0.0 for s in range(8 * page) if s not in set(slots.tolist()))
    assert (gate is None) == (gates == 0) and (gate is None or rel_err(gate, torch.sigmoid(x[:, Rq + Kv + R:])) < 1e-6)
    q = rnd(T, H * (D + R), seed=4).float()
    plain, row = K.latent_queries(q.cuda(), pos.cuda(), *tables(rot), H, D, R, Kv, dtype)
    qv = q.double().view(T, H, D + R)
    assert rel_err(plain, qv[..., :D]) < tol and rel_err(row[..., Kv:], P.turn_neighbours(qv[..., D:], pos, rot)) < tol


# ---------------------------------------------------------------------------------------- router and experts
@pytest.mark.parametrize("E,top,groups", [(20, 3, (2, 1)), (12, 4, (4, 2)), (6, 1, (1, 1)), (4, 4, (2, 2)), (1, 1, (1, 1)), (64, 6, (16, 3)), (40, 40, (1, 1)), (258, 33, (6, 1))])
def test_softmax_router_over_all_experts(K, E, top, groups):
    T = 70
    logits, corr = rnd(T, E, seed=E, scale=2.5).float(), rnd(E, seed=top, scale=0.2).float()
    chosen, weights, gate = K.moe_route_top(logits.cuda(), corr.cuda(), E, top, *groups, 1e-20, scoring="softmax_all", group_score="max")
    w = {"router": torch.eye(E, dtype=F64), "correction": corr.double()}
    want_c, want_w = P.route(logits.double(), w, "", {"experts": E, "top": top, "groups": {"count": groups[0], "keep": groups[1]}})
    assert gate is None and torch.equal(chosen.cpu().sort(-1).values.long(), want_c.sort(-1).values)
    a, b = chosen.cpu().long().argsort(-1), want_c.argsort(-1)
    assert rel_err(weights.cpu().gather(1, a), want_w.gather(1, b)) < 1e-5


@BOTH
@pytest.mark.parametrize("T,width,ff,E,identity,top", [(1, 48, 24, 5, 3, 2), (9, 44, 9, 4, 1, 4), (70, 384, 88, 12, 4, 3), (300, 64, 40, 3, 2, 1), (260, 192, 96, 12, 12, 4),
                                                       (130, 44, 9, 1, 7, 2)])
def test_identity_experts(K, dtype, T, width, ff, E, identity, top):
    """Few tokens (weights streamed per token) and many (sorted by expert, grouped products), some of whose choices all are the
    identity and some none; without the option such numbers add nothing."""
    x = rnd(T, width, seed=1).to(dtype)
    gu, down = rnd(E, 2 * ff, width, seed=2, scale=width ** -0.5).to(dtype), rnd(E, width, ff, seed=3, scale=ff ** -0.5).to(dtype)
    g = torch.Generator().manual_seed(4)
    chosen = torch.stack([torch.randperm(E + identity, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    weights, add = torch.rand(T, top, generator=g), rnd(T, width, seed=5).float()
    for on in (True, False):
        got = K.moe_experts(x.cuda(), chosen.cuda(), gu.cuda(), down.cuda(), 1.0, add=add.cuda(), out_dtype=torch.float32, weights=weights.cuda(), identity=on)
        want = add.double().clone()
        for e in range(E + identity if on else E):
            t, j = torch.nonzero(chosen == e, as_tuple=True)
            if len(t):
                w = {"gate": gu[e, :ff].double(), "up": gu[e, ff:].double(), "down": down[e].double()} if e < E else None
                want[t] += weights[t, j].double()[:, None] * (P.gated_expert(x[t].double(), w, "") if e < E else x[t].double())
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
    """Sizes off every fast path (see lefolorn_tools.odd_shapes), whole prompts and the mixed schedule."""
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
    """A short prompt, then 400 tokens one by one (graphs): windows pass over decoded tokens, window pages come back, distances
    pass every row of the tables; the logits equal those of the whole sequence."""
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
