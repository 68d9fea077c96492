"""The Sozudra design on the engine's host side, without a GPU: configuration, tensor names, the plain mechanisms
themselves, and the real step function, cache manager, scheduler, trace replay and entry point driven with the torch
stand-ins for the kernels (emulated_kernels.py) against the plain implementation (plain_sozudra.py).  What is checked here is
the bookkeeping - a cache and a state per pass over a looped layer, two members of a mixer with a cache and a state each,
the previous token as state, window pages that come back while a request runs, pages and slots used again, portions cut
anywhere; the kernels themselves are checked by the GPU tests."""
import io
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import plain_sozudra as P
import sozudra_tools as X
import trace_tools as TT
from emulated_kernels import EmulatedKernels
from model_tools import random_requests

from rvllm_b200 import ConfigError, LLM, SamplingParams, config_from_dict, kernels as kernel_pkg, load_config
from rvllm_b200.engine import trace as trace_mod
from rvllm_b200.engine.step import StepEntry
from rvllm_b200.models.decoder import DecoderModel, expected_tensors
from rvllm_b200.parts.base import CompositeNeed, KvCacheNeed, StateNeed
from rvllm_b200.parts.rope import RotaryEncoding

F64 = torch.float64


@pytest.fixture
def emulated():
    kernel_pkg.set_library(EmulatedKernels())
    yield
    kernel_pkg.set_library(None)


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


# ---------------------------------------------------------------------------------------- configuration
def test_config_round_trip_and_spec():
    for make in (X.small_a, X.small_b, X.odd_shapes):
        cfg = config_from_dict(make())
        assert config_from_dict(cfg.to_dict()) == cfg and not cfg.to_spec().validate()
    cfg = config_from_dict(X.small_a())
    spec = cfg.to_spec()
    assert spec.residual_dtype == "float32" and spec.lm_head_name == "head"
    # the span 1..2 runs three times; every run has a cache slot of its own
    assert [(e.layer, e.cache) for e in spec.run_order] == [(0, 0), (1, 1), (2, 2), (1, 3), (2, 4), (1, 5), (2, 6), (3, 7), (4, 8)]
    assert cfg.run_plan() == P.layer_order(X.small_a())
    shapes = {n: ts.shape for n, ts in expected_tensors(spec).items()}
    assert shapes["bigram"] == (38, 48) and shapes["head"] == (131, 48) and shapes["final.norm"] == (48,) and shapes["l4.norm1"] == (48,)
    assert shapes["l0.mix.q"] == (144, 48) and shapes["l0.mix.q.b"] == (144,) and shapes["l0.mix.k"] == (48, 48) and shapes["l0.mix.v.b"] == (40,)
    assert shapes["l0.mix.lq1"] == (12,) and shapes["l0.mix.lk2"] == (12,) and shapes["l0.mix.o"] == (48, 120) and "l0.mix.o.b" not in shapes
    assert shapes["l1.mix.left.q"] == (96, 48) and shapes["l1.mix.left.v"] == (32, 48) and shapes["l1.mix.left.o"] == (48, 64)
    assert "l1.mix.left.q.b" not in shapes and shapes["l1.mix.right.z"] == (40, 48) and shapes["l1.mix.right.x.b"] == (40,)
    assert shapes["l1.mix.right.o"] == (48, 40) and "l1.mix.right.g.b" not in shapes
    assert shapes["l0.mlp.router"] == (6, 48) and shapes["l0.mlp.router.b"] == (6,) and shapes["l0.mlp.shared.sg"] == (1, 48)
    assert shapes["l0.mlp.e5.gate"] == (24, 48) and shapes["l0.mlp.e5.down"] == (48, 24) and "l0.mlp.e6.up" not in shapes
    assert "l1.mlp.shared.up" not in shapes and "l3.norm2" not in shapes and "l3.mlp.router" not in shapes
    needs = DecoderModel(spec).cache_needs()
    # two maps side by side in a key row, the slot a multiple of 16
    assert needs[0] == KvCacheNeed(2, 32, 13) and needs[8] == KvCacheNeed(1, 48, 7)
    assert needs[1] == CompositeNeed((KvCacheNeed(2, 32, 11), StateNeed((40,), "float32")))
    assert needs[9] == StateNeed((1,), "int32") and sorted(needs) == list(range(10))       # the previous token
    none = config_from_dict(X.odd_shapes()).to_spec()
    assert not none.embedding_hooks and sorted(DecoderModel(none).cache_needs()) == [0, 1, 2, 3]
    assert "bigram" not in expected_tensors(none)


def test_config_errors_are_collected():
    bad = X.small_a()
    bad["layers"][0]["mixer"]["kv_heads"] = 4                # 6 heads on 4
    bad["layers"][1]["mixer"]["left"]["vdim"] = 15           # does not turn in pairs
    bad["layers"][2]["mixer"]["rot"]["dims"] = 10            # beyond the head
    bad["layers"][2]["mlp"]["router"]["top"] = 9
    bad["layers"][3]["type"] = "mlstm"
    del bad["layers"][4]["mixer"]["rot"]["scaling"]["fast"]
    bad["loop"]["stop"] = 9
    bad["embedding"]["bigram"]["buckets"] = 0
    del bad["residual_mult"]
    with pytest.raises(ConfigError) as e:
        config_from_dict(bad)
    text = str(e.value)
    for piece in ("layers[0]", "layers[1]: left", "layers[2]", "`top`", "layers[3]", "rot.scaling", "loop", "buckets", "residual_mult"):
        assert piece in text, (piece, text)
    for empty in (None, {}):
        ok = X.odd_shapes()
        ok["embedding"] = empty
        assert config_from_dict(ok).bigram is None
    looped = X.small_b()
    looped["loop"] = {"start": 1, "stop": 1, "times": 4}      # an empty span
    assert config_from_dict(looped).run_plan() == [0, 1]


# ---------------------------------------------------------------------------------------- the plain mechanisms
def test_plain_rotation_and_its_scaling():
    rot = {"dims": 6, "base": 50.0}
    v, pos = rnd(5, 2, 8), torch.tensor([0, 3, 4, 9, 100])
    out = P.turn_halves(v, pos, rot)
    assert torch.equal(out[0], v[0]) and torch.equal(out[..., 6:], v[..., 6:])
    ang = 3.0                                                                          # pair 0 turns by the position itself
    assert torch.allclose(out[1, 0, 0], v[1, 0, 0] * math.cos(ang) - v[1, 0, 3] * math.sin(ang))
    assert torch.allclose(out[1, 0, 3], v[1, 0, 3] * math.cos(ang) + v[1, 0, 0] * math.sin(ang))
    assert torch.allclose(P.turn_halves(out, -pos, rot), v)                            # and back
    # the scaling: the fastest pairs keep their frequency, the slowest have it divided, all elements grow alike
    scaled = {"dims": 32, "base": 10000.0, "scaling": {"factor": 8.0, "original": 1024, "fast": 32.0, "slow": 1.0}}
    plain = [10000.0 ** (-2.0 * i / 32) for i in range(16)]
    got = [P.pair_frequency(i, scaled) for i in range(16)]
    assert got[0] == plain[0] and abs(got[15] - plain[15] / 8.0) < 1e-15
    assert all(plain[i] / 8.0 - 1e-15 <= got[i] <= plain[i] + 1e-15 for i in range(16)) and got == sorted(got, reverse=True)
    assert sum(1 for i in range(16) if plain[i] / 8.0 < got[i] < plain[i]) >= 3         # the ramp between
    # which pair turns 32 times over 1,024 positions: 1,024 f = 32 * 2 pi
    lo = 32 * math.log(1024 / (2 * math.pi * 32)) / (2 * math.log(10000.0))
    assert got[math.floor(lo)] == plain[math.floor(lo)] and got[math.floor(lo) + 1] < plain[math.floor(lo) + 1]
    x = rnd(4, 32, seed=2)
    grown = P.turn_halves(x, torch.arange(4), scaled)
    assert torch.allclose(grown.norm(dim=-1), x.norm(dim=-1) * (0.1 * math.log(8.0) + 1.0))


@pytest.mark.parametrize("scaling", [None, {"factor": 4.0, "original": 64, "fast": 16.0, "slow": 1.5}, {"factor": 1.0, "original": 100, "fast": 2.0, "slow": 2.0},
                                     {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0}])
@pytest.mark.parametrize("dims,base", [(24, 500.0), (6, 40.0), (128, 1e6), (2, 9.0)])
def test_rotation_tables(dims, base, scaling):
    enc = RotaryEncoding(dims, base, None if scaling is None else dict(scaling, rope_type="yarn"), dims)
    enc.prepare(300, "cpu")
    cos, sin = enc.rotation_tables()
    one = torch.zeros(300, dims, dtype=F64)
    one[:, :dims // 2] = 1.0
    want = P.turn_halves(one, torch.arange(300), {"dims": dims, "base": base, "scaling": scaling})
    assert float((cos - want[:, :dims // 2]).abs().max()) < 3e-5 and float((sin - want[:, dims // 2:]).abs().max()) < 3e-5


def test_plain_turned_values_depend_on_distances_alone():
    """Shifting every position leaves the layer's result unchanged; a value that is not turned (or not turned back) would not."""
    m = {"heads": 2, "kv_heads": 1, "dim": 6, "vdim": 4, "scale": 0.5, "softcap": 3.0, "mask": {"size": 5}, "rot": {"dims": 4, "base": 20.0}}
    w = {"q": rnd(12, 9, seed=1), "k": rnd(6, 9, seed=2), "v": rnd(4, 9, seed=3), "o": rnd(9, 8, seed=4)}
    h = rnd(11, 9, seed=5)
    a = P.turned_value_attention(h, w, "", m, 1e-5, torch.arange(11))
    b = P.turned_value_attention(h, w, "", m, 1e-5, torch.arange(11) + 37)
    assert torch.allclose(a, b, atol=1e-10)
    # the first token sees itself only: its value comes back as projected
    assert torch.allclose(a[0], torch.cat([w["v"] @ h[0]] * 2) @ w["o"].T)
    # with one key in the window every result is the token's own value, but its score cannot matter
    own = P.turned_value_attention(h, w, "", dict(m, mask={"size": 1}), 1e-5, torch.arange(11))
    assert torch.allclose(own, torch.cat([h @ w["v"].T] * 2, dim=1) @ w["o"].T)
    # scaling a token's input leaves its key as it is (unit norm)
    h2 = h.clone()
    h2[7] *= 3.0
    keys = lambda hh: P.unit_rms(P.turn_halves((hh @ w["k"].T).reshape(11, 1, 6), torch.arange(11), m["rot"]), 0.0)
    assert torch.allclose(keys(h), keys(h2))


def test_plain_window_edge_and_cap():
    q = torch.ones(1, 1, dtype=F64).expand(12, 1)
    k = torch.zeros(12, 1, dtype=F64)
    k[3] = 50.0
    wts = P.visible_weights(q, k, torch.arange(12), 1.0, None, 6)
    assert float(wts[8, 3]) > 0.999 and float(wts[9, 3]) == 0.0 and float(wts[3, 3]) > 0.999 and float(wts[2, 3]) == 0.0
    assert torch.allclose(wts[9, 4:10], torch.full((6,), 1 / 6, dtype=F64))
    capped = P.visible_weights(q, k, torch.arange(12), 1.0, 2.0, 6)
    assert abs(float(capped[8, 3]) - math.exp(2.0) / (math.exp(2.0) + 5.0)) < 1e-9
    assert float(P.visible_weights(q, k, torch.arange(12), 1.0, None, None)[11, 3]) > 0.999


def test_plain_differential_maps():
    m = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 6, "scale": 0.5, "diff": 0.3, "mask": {"size": 100}, "rot": {"dims": 2, "base": 20.0}}
    w = {"q": rnd(16, 9, seed=1), "k": rnd(8, 9, seed=2), "v": rnd(6, 9, seed=3), "o": torch.eye(12, dtype=F64),
         "q.b": rnd(16, seed=5), "k.b": rnd(8, seed=6), "v.b": rnd(6, seed=7)}
    for n, s in (("lq1", 8), ("lk1", 9), ("lq2", 10), ("lk2", 11)):
        w[n] = rnd(4, seed=s) * 0.5
    lam = P.map_difference(w, "", 0.3)
    assert abs(lam - (math.exp(float(w["lq1"] @ w["lk1"])) - math.exp(float(w["lq2"] @ w["lk2"])) + 0.3)) < 1e-12
    h = rnd(5, 9, seed=12)
    out = P.differential_attention(h, w, "", m, 0.0, torch.arange(5)).view(5, 2, 6)
    # unit RMS per head times 1 - diff; the first token: both maps are its own value
    assert torch.allclose((out * out).mean(-1).sqrt(), torch.full((5, 2), 0.7, dtype=F64))
    v0 = w["v"] @ h[0] + w["v.b"]
    sign = 1.0 if lam < 1.0 else -1.0
    assert torch.allclose(out[0, 0], 0.7 * sign * v0 / (v0 * v0).mean().sqrt())
    # without the second map (lambda 0) it is the first map alone
    zero = dict(w, lq1=torch.zeros(4, dtype=F64), lq2=torch.zeros(4, dtype=F64))
    assert P.map_difference(zero, "", 0.0) == 0.0


def test_plain_min_gru_against_the_closed_form():
    w = {n: rnd(3, 5, seed=i) for i, n in enumerate(("z", "x", "g"))}
    w.update({"z.b": rnd(3, seed=7), "x.b": rnd(3, seed=8), "o": torch.eye(3, dtype=F64)})
    h = rnd(6, 5, seed=9)
    got = P.min_gru(h, w, "", {"width": 3})
    z = torch.sigmoid(h @ w["z"].T + w["z.b"])
    u = h @ w["x"].T + w["x.b"]
    c = torch.where(u >= 0, u + 0.5, 1.0 / (1.0 + torch.exp(-u)))
    for t in range(6):
        S = sum(z[j] * c[j] * torch.prod(1.0 - z[j + 1:t + 1], dim=0) for j in range(t + 1))
        g = h[t] @ w["g"].T
        assert torch.allclose(got[t], S * torch.nn.functional.silu(g))
    assert bool((u < 0).any()) and bool((u >= 0).any())


def test_plain_router_and_bigram():
    w = {"router": torch.zeros(5, 2, dtype=F64), "router.b": torch.tensor([0.0, 0.0, 3.0, 0.0, 0.0], dtype=F64)}
    w["router"][:, 0] = torch.tensor([2.0, 1.0, -1.5, 0.0, 1.7])
    chosen, weights = P.route(torch.ones(1, 2, dtype=F64), w, "", {"experts": 5, "top": 3})
    assert chosen[0].tolist() == [0, 4, 2]                      # the bias lifts expert 2 over expert 1, and counts in its weight
    e = torch.exp(torch.tensor([2.0, 1.7, 1.5], dtype=F64))
    assert torch.allclose(weights[0], e / e.sum())
    table = {"embed": torch.zeros(9, 1, dtype=F64), "bigram": torch.arange(8, dtype=F64)[:, None]}
    x = P.embed(torch.tensor([4, 2, 2, 8]), table, {"buckets": 7, "mul_prev": 3, "mul_cur": 5})
    assert x[:, 0].tolist() == [7.0, float((4 * 3 + 2 * 5) % 7), float((2 * 3 + 2 * 5) % 7), float((2 * 3 + 8 * 5) % 7)]


# ---------------------------------------------------------------------------------------- replay through the engine
LENGTHS = (41, 70, 23, 88, 1, 37)
SCHEDULES = {"whole": TT.schedule_whole, "bulk_tail": TT.schedule_bulk_tail, "portions": TT.schedule_portions,
             "mixed": TT.schedule_mixed}
_cache = {}


def _reference(which):
    if which not in _cache:
        folder = X.write_folder({"a": X.small_a, "b": X.small_b, "odd": X.odd_shapes}[which](), seed=5, edit=X.lively)
        vocab = load_config(folder).vocab_size
        reqs = random_requests(vocab, LENGTHS, seed=4)
        _cache[which] = (folder, vocab, reqs, X.plain_logits(folder, reqs))
    return _cache[which]


@pytest.mark.parametrize("which", ["a", "odd"])
@pytest.mark.parametrize("schedule", list(SCHEDULES))
def test_replay_matches_plain_under_every_cut(emulated, tmp_path, which, schedule):
    folder, vocab, reqs, ref = _reference(which)
    trace = SCHEDULES[schedule](reqs)
    if schedule == "portions":
        assert min(len(e["tokens"]) for s in trace.steps for e in s["entries"]) <= 2
    if schedule == "mixed":
        assert max(len(s["entries"]) for s in trace.steps) == 4 and trace.preemptions == 1     # pages and slots are used again
    engine = trace_mod.build_engine(folder, "float32", trace.max_tokens, block_size=8, device="cpu")
    n = trace_mod.replay(engine, io.StringIO(trace.lines()), str(tmp_path), io.StringIO())
    assert n == len(trace.steps)
    got = TT.read_logits(str(tmp_path), trace, vocab)
    assert TT.compare(got, ref, 3e-5, f"{which}/{schedule}") < 3e-5
    engine.cache.check()
    assert not engine.cache.requests and engine.cache.slots.num_free == 4


def test_streams_after_every_layer(emulated):
    folder, vocab, reqs, _ = _reference("a")
    cfg, w = X.read_folder(folder)
    toks = reqs["r2"]
    want = []
    P.forward(cfg, w, toks, streams=want)
    engine = trace_mod.build_engine(folder, "float32", 64, block_size=8, device="cpu")
    seen = []

    def recording(block):
        def run(x, ctx, cache, write=True):
            y = block(x, ctx, cache, write)
            seen.append(y.clone())           # (the next layer adds into y in place)
            return y
        return run

    for layer in engine.model.layers:
        layer.block = recording(layer.block)
    engine.runner.step([StepEntry("x", toks, [0])])
    assert len(seen) == len(want) == 9
    for k, (a, b) in enumerate(zip(seen, want)):
        assert float((a.double() - b).abs().max() / b.abs().max()) < 1e-5, f"layer run {k}"


def test_norms_travel_to_the_next_layer(emulated):
    """Each run's inputs but the first's are formed by the run before it, in the kernel that writes the stream; a block of
    another kind behind it, or one behind a hook, gets none."""

    class Recording(EmulatedKernels):
        calls = []

        def stream_combine(self, x, terms, norms, out_dtype):
            self.calls.append((len(terms), len(norms)))
            return super().stream_combine(x, terms, norms, out_dtype)

    kernel_pkg.set_library(Recording())
    folder, vocab, reqs, ref = _reference("a")
    engine = trace_mod.build_engine(folder, "float32", 64, block_size=8, device="cpu")
    engine.runner.step([StepEntry("x", reqs["r2"][:5], [4])])
    # before layer 0: both norms; then per run its terms (mixer or two members, experts) and the norms of the next run
    assert Recording.calls == [(0, 2), (2, 2), (3, 2), (2, 2), (3, 2), (2, 2), (3, 2), (2, 1), (2, 1), (1, 0)]


def test_window_pages_come_back_and_states_start_at_zero(emulated):
    folder, vocab, reqs, ref = _reference("a")
    engine = trace_mod.build_engine(folder, "float32", 192, block_size=8, device="cpu")
    cache = engine.cache
    windows = sorted((g.need.window or 0) for g in cache.groups)
    assert windows == [0, 7, 11, 13, 29]
    at = [i for i, g in enumerate(cache.groups) if g.need.window == 11]
    assert len(cache.groups[at[0]].cache_slots) == 3                       # one per pass
    toks = reqs["r3"]
    rows = [engine.runner.step([StepEntry("x", toks[:50], list(range(50)))])]
    table = cache.block_table("x", at[0])
    assert table[:5] == [-1] * 5 and table[5] >= 0                         # keys below 50 - 11 + 1 = 40 are gone: pages 0 to 4
    for p in range(50, len(toks)):
        rows.append(engine.runner.step([StepEntry("x", toks[p:p + 1], [0])]))
    got = torch.cat(rows).double()
    assert float((got - ref["r3"]).abs().max() / ref["r3"].abs().max()) < 3e-5
    assert int(cache.view(9).state[cache.state_slot("x"), 0]) == toks[-1]  # the previous token is state
    engine.runner.finish("x")
    # the slot's state rows hold what the request left; the next request in the same slot starts from zeros all the same
    states = list(cache._state.values())
    assert len(states) == 5 and all(float(t[0].abs().max()) > 0 for t in states)       # three passes, the last layer pair's, the token
    again = engine.runner.step([StepEntry("y", reqs["r0"], list(range(len(reqs["r0"]))))]).double()
    assert cache.state_slot("y") == 0
    assert float((again - ref["r0"]).abs().max() / ref["r0"].abs().max()) < 3e-5
    engine.runner.finish("y")
    cache.check()


def test_generate_greedy_matches_plain(emulated):
    folder, vocab, reqs, ref = _reference("a")
    cfg, w = X.read_folder(folder)
    prompts = [reqs["r2"], reqs["r4"], reqs["r0"][:30]]
    llm = LLM(folder, dtype="float32", device="cpu", block_size=8, num_blocks=24, max_model_len=64, max_num_seqs=2,
              max_num_batched_tokens=16, max_prefill_chunk=7)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.outputs[0].token_ids == P.greedy(cfg, w, p, 6)
    assert not llm.engine.cache.requests


def test_command_line_info_and_random_weights(tmp_path):
    """`rvllm random-weights` writes a folder for the design from a config.json; `rvllm info` reads it back."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg_file = tmp_path / "config.json"
    cfg_file.write_text(json.dumps(X.small_a()))
    out = tmp_path / "model"
    run = lambda *a: subprocess.run([sys.executable, os.path.join(root, "bin", "rvllm"), *a], capture_output=True, text=True, timeout=300)
    p = run("random-weights", "--config", str(cfg_file), "--out", str(out), "--seed", "3")
    assert p.returncode == 0, p.stderr
    p = run("info", "--model", str(out))
    assert p.returncode == 0, p.stderr
    info = json.loads(p.stdout)
    assert info["architecture"] == "Sozudra" and info["config"]["layers"][1]["mixer"]["right"]["width"] == 40
    cfg, w = X.read_folder(str(out))
    assert P.forward(cfg, w, [1, 2, 3]).shape == (3, 131)
