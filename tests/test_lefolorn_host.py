"""The Lefolorn design on the engine's host side, without a GPU: configuration, tensor names, the plain mechanisms themselves,
and the real step function, cache manager, scheduler, trace replay and entry point driven with the torch stand-ins for the
kernels (emulated_kernels.py) against the plain implementation (plain_lefolorn.py).  What is checked here is the bookkeeping -
groups of layers with a window, without one and with one row per token, values that travel between the layers of a step,
window pages that come back while a request runs, pages used again, portions cut anywhere; the kernels themselves are checked
by the GPU tests."""
import io
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import lefolorn_tools as X
import plain_lefolorn as P
import trace_tools as TT
from emulated_kernels import EmulatedKernels
from model_tools import random_requests

from rvllm_b200 import ConfigError, LLM, SamplingParams, config_from_dict, kernels as kernel_pkg, load_config
from rvllm_b200.engine import trace as trace_mod
from rvllm_b200.engine.step import StepEntry
from rvllm_b200.errors import LoaderError
from rvllm_b200.models.decoder import DecoderModel, expected_tensors
from rvllm_b200.parts.base import KvCacheNeed
from rvllm_b200.parts.distance import bucket_rows, distance_table
from rvllm_b200.weights import WeightSource

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
    shapes = {n: ts.shape for n, ts in expected_tensors(spec).items()}
    assert shapes["l0.norm1"] == shapes["l0.ls1"] == shapes["l0.ls2"] == shapes["l0.rg2.b"] == (48,) and shapes["l0.rg1"] == (48, 48)
    assert "l0.norm2" not in shapes and shapes["l0.mix.q"] == (72, 48) and shapes["l0.mix.v.b"] == (40,) and shapes["l0.mix.k.norm"] == (12,)
    assert shapes["l0.mix.o"] == (48, 120) and not {"l0.mix.rel", "l0.mix.g", "l0.mix.vmix"} & set(shapes)
    assert shapes["l1.mix.rel"] == (12, 4) and shapes["l1.mix.g"] == (64, 48) and shapes["l1.mix.vmix"] == () and "l1.mix.g.b" not in shapes
    assert shapes["l2.mix.dq"] == (18, 48) and shapes["l2.mix.uq"] == (100, 18) and shapes["l2.mix.dkv"] == (28, 48)
    assert shapes["l2.mix.dq.norm"] == (18,) and shapes["l2.mix.uk"] == (70, 22) and shapes["l2.mix.uv"] == (50, 22) and shapes["l2.mix.sink"] == (5,)
    assert "l2.mix.q" not in shapes
    # the router also has an output (and a correction) per identity expert, which has no tensors
    assert shapes["l0.mlp.router"] == (8, 48) and shapes["l0.mlp.correction"] == (8,) and "l0.mlp.e5.gate" in shapes and "l0.mlp.e6.gate" not in shapes
    assert shapes["l0.mlp.shared.down"] == (48, 16) and "l0.mlp.shared.sg" not in shapes and "l1.mlp.shared.up" not in shapes
    # a layer without a feed-forward has nothing to scale or gate behind one; a checkpoint may hold such tensors all the same
    assert "l3.ls1" in shapes and not {"l3.ls2", "l3.rg2", "l3.rg2.b", "l3.mlp.router"} & set(shapes)
    assert {"l3.ls2", "l3.rg2", "l3.rg2.b"} <= set(spec.ignored_tensors)
    needs = DecoderModel(spec).cache_needs()
    assert needs[0] == KvCacheNeed(2, 32, 13) and needs[1] == KvCacheNeed(2, 32, None) and needs[3] == KvCacheNeed(2, 16, 7)
    assert needs[2] == KvCacheNeed(1, 28, None, planes=1) and needs[4] == KvCacheNeed(1, 27, None, planes=1)
    # which layer's values the others take a share of
    roles = [layer.parts["mixer"].params.get("value_mix") for layer in spec.layers]
    assert roles == [None, "first", None, "later", None, "later"]


def test_config_errors_are_collected():
    bad = X.small_a()
    bad["norm"]["groups"] = 5                                # 48 columns
    bad["layers"][0]["mixer"]["kv_heads"] = 4                # 6 heads on 4
    bad["layers"][0]["mlp"]["router"]["groups"]["count"] = 3 # 8 outputs
    bad["layers"][1]["mixer"]["q_temp"]["every"] = 0
    bad["layers"][2]["mixer"]["rot"]["dims"] = 8             # beyond the rotated part
    del bad["layers"][2]["mixer"]["q_rank"]
    bad["layers"][3]["mixer"]["vdim"] = 17                   # 34 elements take no share of 32
    bad["layers"][4]["type"] = "mlstm"
    bad["layers"][5]["mixer"]["v_mix"] = 1
    with pytest.raises(ConfigError) as e:
        config_from_dict(bad)
    text = str(e.value)
    for piece in ("norm: ", "layers[0]", "equal groups", "q_temp", "layers[2]: `rot.dims`", "q_rank", "layers[3]: `v_mix`", "layers[4]", "layers[5]: `v_mix`"):
        assert piece in text, (piece, text)
    with pytest.raises(ConfigError):
        bucket_rows(12, 6)                                   # the logarithmic rows need a limit beyond the first half's


def test_the_checkpoint_says_how_many_rows_a_distance_table_has(emulated):
    """The folder is written with 12 rows; a configuration that names none (its default is another number) reads it all the same.
    Every other size stays checked."""
    folder = X.write_folder(X.small_a(), seed=5, edit=X.lively)
    cfg, w = X.read_folder(folder)
    for layer in cfg["layers"]:
        layer["mixer"].pop("bias_rows", None)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    toks = list(range(3, 60))
    engine = trace_mod.build_engine(folder, "float32", 64, block_size=8, device="cpu")
    got = engine.runner.step([StepEntry("x", toks, list(range(57)))]).double()
    want = P.forward(cfg, w, toks)
    assert float((got - want).abs().max() / want.abs().max()) < 3e-5
    specs = expected_tensors(config_from_dict(cfg).to_spec())
    shapes = {n: ts.shape for n, ts in specs.items()}
    source = WeightSource(folder)
    source.check(shapes, free={n: ts.free for n, ts in specs.items()})
    with pytest.raises(LoaderError):
        source.check(shapes)
    with pytest.raises(LoaderError):
        source.check(dict(shapes, **{"l1.mix.rel": (32, 5)}), free={n: ts.free for n, ts in specs.items()})


# ---------------------------------------------------------------------------------------- the plain mechanisms
def test_plain_norm_in_groups():
    x, w = rnd(3, 12, seed=1), rnd(12, seed=2)
    out = P.grouped_norm(x, w, 3, 1e-3)
    for g in range(3):
        part = x[:, 4 * g:4 * g + 4]
        assert torch.allclose(out[:, 4 * g:4 * g + 4], part / torch.sqrt((part ** 2).mean(-1, keepdim=True) + 1e-3) * w[4 * g:4 * g + 4])
    x2 = x.clone()
    x2[:, :4] *= 9.0                                                # a group's size does not touch the others
    assert torch.equal(P.grouped_norm(x2, w, 3, 1e-3)[:, 4:], out[:, 4:]) and not torch.allclose(P.grouped_norm(x2, w, 1, 1e-3)[:, 4:], out[:, 4:])


@pytest.mark.parametrize("rows,limit", [(32, 250), (32, 128), (12, 40), (5, 9), (2, 3), (3, 60), (7, 3.5), (64, 4096)])
def test_distance_buckets(rows, limit):
    got = bucket_rows(rows, limit)
    assert got == [P.distance_bucket(n, rows, limit) for n in range(len(got))]
    assert all(P.distance_bucket(n, rows, limit) == rows - 1 for n in (len(got), len(got) + 1, 10 * len(got), 10 ** 6))
    half = rows // 2
    assert got[:half] == list(range(half)) and got[half] == half if len(got) > half and rows > 2 else True
    assert got == sorted(got) and got[-1] == rows - 1 and (len(got) < 2 or got[-2] < rows - 1) and len(got) - 1 <= math.ceil(limit)
    table = torch.randn(rows, 6, generator=torch.Generator().manual_seed(rows))
    bias = distance_table(table, limit, 2)
    assert bias.distances == len(got) and bias.heads == 6 and tuple(bias.natural.shape) == (2, len(got), 3)
    for n in (0, 1, len(got) - 1):
        n = min(n, len(got) - 1)
        for h in range(6):
            assert float(bias.natural[h // 3, n, h % 3]) == float(table[got[n], h])
    assert torch.allclose(bias.log2, bias.natural * math.log2(math.e))


def test_plain_temperature_and_sinks():
    pos = torch.tensor([0, 3, 4, 8, 9, 99])
    t = P.query_temperature(pos, {"coef": 0.5, "every": 5})
    assert [round(float(v), 12) for v in t] == [round(1 + 0.5 * math.log(n + 1), 12) for n in (0, 0, 1, 1, 2, 20)]
    assert P.query_temperature(pos, None).tolist() == [1.0] * 6
    q, k = rnd(5, 4, seed=1), rnd(5, 4, seed=2)
    p1 = P.head_weights(q, k, torch.arange(5), 0.7, sink=0.0)
    s = (q @ k.T) * 0.7
    for i in range(5):
        e = torch.exp(s[i, :i + 1])
        assert torch.allclose(p1[i, :i + 1], e / (1.0 + e.sum()))
    p2 = P.head_weights(q, k, torch.arange(5), 0.7, sink=2.0)
    assert torch.allclose(p2[4], torch.exp(s[4]) / (math.exp(2.0) + torch.exp(s[4]).sum()))


def test_plain_distance_bias_and_window_edge():
    q, k = torch.zeros(12, 3, dtype=F64), rnd(12, 3, seed=1)
    table = torch.zeros(6, dtype=F64)
    table[4] = 40.0                                                  # row 4 of 6 with limit 9: distances 5 and 6
    assert [n for n in range(12) if P.distance_bucket(n, 6, 9.0) == 4] == [5, 6]
    w = P.head_weights(q, k, torch.arange(12), 1.0, table=table, limit=9.0)
    assert torch.allclose(w[10, 4:6], torch.tensor([0.5, 0.5], dtype=F64)) and torch.allclose(w[4, :5], torch.full((5,), 0.2, dtype=F64))
    q = torch.ones(12, 1, dtype=F64)
    k = torch.zeros(12, 1, dtype=F64)
    k[3] = 50.0
    w = P.head_weights(q, k, torch.arange(12), 1.0, window=6)
    assert float(w[8, 3]) > 0.999 and float(w[9, 3]) == 0.0 and float(w[3, 3]) > 0.999 and float(w[2, 3]) == 0.0
    capped = P.head_weights(q, k, torch.arange(12), 1.0, cap=2.0, window=6)
    assert abs(float(capped[8, 3]) - math.exp(2.0) / (math.exp(2.0) + 5.0)) < 1e-9


def test_plain_value_mixing():
    m = {"v_mix": True}
    a, b = rnd(4, 2, 3, seed=1), rnd(4, 2, 3, seed=2)
    memory = {}
    assert P.mix_values(b, {}, "", {"v_mix": False}, memory) is b and not memory
    assert P.mix_values(a, {"vmix": torch.tensor(0.9, dtype=F64)}, "", m, memory) is a           # the first one's share is not used
    got = P.mix_values(b, {"vmix": torch.tensor(0.25, dtype=F64)}, "", m, memory)
    assert torch.allclose(got, 0.75 * b + 0.25 * a) and memory["first"] is a                     # ... and stays the first for good


def test_plain_router():
    w = {"router": torch.eye(6, dtype=F64), "correction": torch.tensor([0.0, 0.0, 0.0, 0.0, 0.0, -0.9], dtype=F64)}
    z = torch.tensor([[3.0, 0.0, 0.0, 0.0, 2.0, 2.9]], dtype=F64)
    s = torch.softmax(z, -1)[0]
    chosen, weights = P.route(z, w, "", {"experts": 4, "identity": 2, "top": 2})
    assert chosen[0].tolist() == [0, 4] and torch.allclose(weights[0], s[[0, 4]] / (s[0] + s[4]))    # 5 is the second largest, corrected away
    # two groups of three: the group of 0 wins, its second choice has a negative sum or not
    w["correction"][1] = -0.5
    chosen, weights = P.route(z, w, "", {"experts": 6, "top": 3, "groups": {"count": 2, "keep": 1}})
    assert sorted(chosen[0].tolist()) == [0, 1, 2]               # expert 1's choice score is negative, and still before the closed group
    h = rnd(5, 6, seed=3)
    mlp = {"router": {"experts": 1, "identity": 5, "top": 5}, "shared": None}
    ex = {"e0.gate": torch.zeros(2, 6, dtype=F64), "e0.up": torch.zeros(2, 6, dtype=F64), "e0.down": torch.zeros(6, 2, dtype=F64)}
    out = P.moe(h, {**ex, "router": torch.eye(6, dtype=F64), "correction": torch.zeros(6, dtype=F64)}, "", mlp)
    chosen, weights = P.route(h, {"router": torch.eye(6, dtype=F64), "correction": torch.zeros(6, dtype=F64)}, "", mlp["router"])
    assert torch.allclose(out, h * (weights * (chosen >= 1)).sum(-1, keepdim=True))               # identity experts give their input back


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
    assert len(seen) == len(want) == 6
    for k, (a, b) in enumerate(zip(seen, want)):
        assert float((a.double() - b).abs().max() / b.abs().max()) < 1e-5, f"layer {k}"


def test_norms_travel_to_the_next_layer(emulated):
    """Each layer's input but the first's is formed by the layer before it, in the kernel that writes the stream."""

    class Recording(EmulatedKernels):
        calls = []

        def grouped_rmsnorm(self, x, gamma, eps, groups, out_dtype=None):
            self.calls.append("norm")
            return super().grouped_rmsnorm(x, gamma, eps, groups, out_dtype)

        def gated_combine(self, x, terms, scales, gates, bias, norm, out_dtype):
            out = super().gated_combine(x, terms, scales, gates, bias, norm, out_dtype)
            if norm is not None:
                self.calls.pop()
            self.calls.append((len(terms), norm is not None))
            return out

    kernel_pkg.set_library(Recording())
    folder, vocab, reqs, ref = _reference("a")
    engine = trace_mod.build_engine(folder, "float32", 64, block_size=8, device="cpu")
    engine.runner.step([StepEntry("x", reqs["r2"][:5], [4])])
    # before layer 0, after each layer (the fourth has no feed-forward, the last no layer behind it), before the LM head
    assert Recording.calls == ["norm", (2, True), (2, True), (2, True), (1, True), (2, True), (2, False), "norm"]


def test_window_pages_come_back(emulated):
    folder, vocab, reqs, ref = _reference("a")
    engine = trace_mod.build_engine(folder, "float32", 192, block_size=8, device="cpu")
    cache = engine.cache
    assert sorted((g.need.window or 0) for g in cache.groups) == [0, 0, 0, 0, 7, 13]   # (two latent rows, two sizes of whole heads)
    at = [i for i, g in enumerate(cache.groups) if g.need.window == 13][0]
    toks = reqs["r3"]
    rows = [engine.runner.step([StepEntry("x", toks[:50], list(range(50)))])]
    table = cache.block_table("x", at)
    assert table[:4] == [-1] * 4 and table[4] >= 0                         # keys below 50 - 13 + 1 = 38 are gone: pages 0 to 3
    for p in range(50, len(toks)):
        rows.append(engine.runner.step([StepEntry("x", toks[p:p + 1], [0])]))
    got = torch.cat(rows).double()
    assert float((got - ref["r3"]).abs().max() / ref["r3"].abs().max()) < 3e-5
    engine.runner.finish("x")
    again = engine.runner.step([StepEntry("y", reqs["r0"], list(range(len(reqs["r0"]))))]).double()      # into the pages just given back
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
    assert info["architecture"] == "Lefolorn" and info["config"]["layers"][1]["mixer"]["q_temp"] == {"coef": 0.7, "every": 5}
    cfg, w = X.read_folder(str(out))
    assert P.forward(cfg, w, [1, 2, 3]).shape == (3, 131)
