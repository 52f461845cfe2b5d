"""Ferodra without a GPU: the plain implementation's mechanisms on cases worked out by hand, the configuration reader, the tensor
names, and the engine's host side (a learned vector per run of a repeated stretch, caches of its own per run, key cells that hold
two maps, experts that pass their input on, page and slot reuse, portions, mixed batches, the scheduler's entry point) with the
torch stand-in for the kernels against the plain implementation."""
import json
import math

import pytest
import torch

from helpers import first_bad, max_error, random_tokens, replay_and_collect, trace_mixed, trace_portions, trace_tail, trace_whole
import plain_ferodra as plain
from fake_kernels import FakeKernels
from ferodra_cases import BLOCK_SIZE, CONFIGS, owed, plain_logits, write_case
from iian_b200 import EngineConfig, SchedulerConfig, ops
from iian_b200.config.registry import get_architecture, load_model_config
from iian_b200.engine.engine import Engine
from iian_b200.engine.model import Model, declare_tensors
from iian_b200.engine.replay import TraceReplayer
from iian_b200.models.qwen3 import ConfigError
from iian_b200.parts.base import KVNeed, StateNeed

F64 = torch.float64


# ---- the plain implementation's mechanisms ------------------------------------------------------------
def test_plain_norm_takes_no_statistics():
    w = {"n": torch.tensor([2.0, -1.0], dtype=F64), "n.alpha": torch.tensor(0.5, dtype=F64), "n.b": torch.tensor([0.25, 1.0], dtype=F64)}
    got = plain.tanh_norm(torch.tensor([[3.0, -4.0]], dtype=F64), w, "n")
    assert torch.allclose(got, torch.tensor([[2 * math.tanh(1.5) + 0.25, math.tanh(2.0) + 1.0]], dtype=F64))


def test_plain_rotation_pairs_neighbours_and_passes_the_rest():
    f, m = plain.rotation({"dims": 4, "base": 100.0})
    assert f.tolist() == pytest.approx([1.0, 0.1]) and m == 1.0
    v = torch.tensor([1.0, 2.0, 3.0, 4.0, 5.0], dtype=F64).view(1, 1, 5).repeat(2, 1, 1)
    out = plain.rotate_neighbours(v, torch.tensor([0, 3]), f, 1.5)
    assert torch.allclose(out[0, 0], torch.tensor([1.5, 3.0, 4.5, 6.0, 5.0], dtype=F64))                # position 0: the factor alone
    assert out[1, 0, 0].item() == pytest.approx(1.5 * (math.cos(3) - 2 * math.sin(3)))
    assert out[1, 0, 1].item() == pytest.approx(1.5 * (2 * math.cos(3) + math.sin(3)))
    assert out[1, 0, 2].item() == pytest.approx(1.5 * (3 * math.cos(0.3) - 4 * math.sin(0.3)))
    assert out[1, 0, 4].item() == 5.0


def test_plain_frequencies_follow_the_ramp():
    # dim(8) = 8 ln(64 / 16 pi) / (2 ln 1e4) < 1: lo 0;  dim(1) = 8 ln(64 / 2 pi) / (2 ln 1e4) = 1.008: hi 2
    f, m = plain.rotation({"dims": 8, "base": 10000.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}})
    assert m == pytest.approx(0.1 * math.log(4.0) + 1.0)
    assert f.tolist() == pytest.approx([1.0, 0.1 * (0.5 / 4 + 0.5), 0.01 / 4, 0.001 / 4])
    # fast and slow so close that the ramp is a step: hi - lo = 0 counts as 0.001
    g, _ = plain.rotation({"dims": 8, "base": 10000.0, "scaling": {"factor": 2.0, "original": 2 * math.pi * 10000.0, "fast": 1e4, "slow": 1e4}})
    assert g.tolist() == pytest.approx([1.0, 0.1 / 2, 0.01 / 2, 0.001 / 2])


def test_plain_attention_subtracts_the_second_map_before_the_norm():
    # two keys; map 1 looks at both alike, map 2 at the second alone (a large score)
    q = torch.tensor([[[[0.0], [1.0]]]], dtype=F64)                                       # [1, 1, 2, 1]
    k = torch.tensor([[[[5.0], [0.0]]], [[[7.0], [1000.0]]]], dtype=F64)
    v = torch.tensor([[[1.0, 0.0]], [[0.0, 3.0]]], dtype=F64)
    o = plain.map_difference(q, k, v, 1.0, None, 0.5, 0.2, 0.0, q_pos0=1)
    d = torch.tensor([0.5, 1.5 - 0.5 * 3.0], dtype=F64)                                    # (a1) - 0.5 (a2 = the second value)
    assert torch.allclose(o[0, 0], d / torch.sqrt((d * d).mean()) * 0.8)
    assert plain.capped_attention(q[:, 0, 1], k[:, 0, 1], v[:, 0], 1.0, 2.0, 1)[0, 1].item() == pytest.approx(
        3 * math.exp(2) / (math.exp(2) + 1))                                               # the cap brings 1000 down to 2
    w = {"lq1": torch.tensor([1.0, 2.0], dtype=F64), "lk1": torch.tensor([0.5, 0.25], dtype=F64),
         "lq2": torch.tensor([1.0, 0.0], dtype=F64), "lk2": torch.tensor([0.3, 9.0], dtype=F64)}
    assert float(plain.map_weight(w, "", 0.2)) == pytest.approx(math.exp(1.0) - math.exp(0.3) + 0.2)


def test_plain_convolution_reads_backwards_and_takes_up_a_cut():
    x = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    taps = torch.tensor([[2.0, 3.0, 5.0]], dtype=F64)                                      # the last column is the current token's
    y = plain.short_convolution(x, taps)
    assert y[:, 0].tolist() == [5.0, 53.0, 532.0]
    assert torch.allclose(plain.short_convolution(x[2:], taps, x[:2]), y[2:])


def test_plain_delta_rule_first_steps_by_hand():
    q = torch.tensor([[[1.0, 1.0]], [[1.0, 0.0]]], dtype=F64)
    k = torch.tensor([[[2.0, 0.0]], [[1.0, 1.0]]], dtype=F64)
    v = torch.tensor([[[5.0]], [[7.0]]], dtype=F64)
    beta, g = torch.tensor([[0.5], [1.0]], dtype=F64), torch.tensor([[0.9], [0.1]], dtype=F64)
    o, S = plain.delta_scan(q, k, v, beta, g)
    assert o[0, 0, 0].item() == pytest.approx(2 * 2.5)                                     # u = 0.5 * 5, S = k u, the read-out sees it
    u = 7 - 0.1 * 5.0                                                                      # the decay comes before the prediction
    assert S[0, :, 0].tolist() == pytest.approx([0.5 + u, u])
    assert o[1, 0, 0].item() == pytest.approx(0.5 + u)
    o2, S2 = plain.delta_scan(q[1:], k[1:], v[1:], beta[1:], g[1:], state=torch.tensor([[[5.0], [0.0]]], dtype=F64))
    assert torch.allclose(o2[0], o[1]) and torch.allclose(S2, S)


def test_plain_router_chooses_with_the_correction_and_weighs_without():
    w = {"router": torch.eye(3, dtype=F64), "correction": torch.tensor([0.0, 0.0, 5.0], dtype=F64)}
    h = torch.log(torch.tensor([[1.0, 3.0, 4.0]], dtype=F64))                               # softmax 1/8, 3/8, 4/8
    ids, wts = plain.router_choice(h, w, "", 2, 1.5)
    assert ids.tolist() == [[2, 1]] and wts[0].tolist() == pytest.approx([1.5 * 0.5, 1.5 * 0.375])
    w["correction"] = torch.tensor([0.5, 0.0, 0.0], dtype=F64)
    ids, wts = plain.router_choice(h, w, "", 2, 1.0)
    assert ids.tolist() == [[0, 2]] and wts[0].tolist() == pytest.approx([0.125, 0.5])      # not renormalised


def test_plain_identity_outputs_pass_the_input_on():
    w = {"router": torch.zeros(3, 2, dtype=F64), "correction": torch.tensor([0.0, 0.0, 9.0], dtype=F64),
         "e0.up": torch.eye(2, dtype=F64), "e0.down": 2 * torch.eye(2, dtype=F64), "e1.up": torch.eye(2, dtype=F64), "e1.down": torch.eye(2, dtype=F64),
         "shared.up": torch.eye(2, dtype=F64), "shared.down": torch.eye(2, dtype=F64), "shared.sg": torch.zeros(1, 2, dtype=F64)}
    h = torch.tensor([[3.0, -2.0]], dtype=F64)
    cfg = {"router": {"experts": 2, "identity": 1, "top": 2, "scale": 3.0}, "shared": {"ff": 2}}
    out = plain.experts_feed_forward(cfg, w, "", h)                                         # output 2 is the identity; then expert 0
    assert out[0].tolist() == pytest.approx([3.0 + 2 * 9.0 + 0.5 * 9.0, -2.0])


def test_plain_run_order_counts_every_run():
    cfg = {"layers": [0, 1, 2, 3], "loop": {"start": 1, "stop": 3, "times": 3}}
    assert plain.run_order(cfg) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert plain.run_order({"layers": [0, 1]}) == [(0, None), (1, None)]


# ---- configuration, names, caches ------------------------------------------------------------------------
def test_config_round_trip_and_registry():
    arch = get_architecture("Ferodra")
    for name, raw in CONFIGS.items():
        c = arch.load_config(raw)
        assert arch.load_config(arch.config_to_dict(c)) == c, name
        spec = arch.build_spec(c)
        spec.validate()
        assert [call.layer for call in spec.order] == [i for i, _ in plain.run_order(raw)]
        assert [(call.turn if call.before is not None else None) for call in spec.order] == [t for _, t in plain.run_order(raw)]
        assert len({call.cache for call in spec.order}) == len(spec.order)            # every run has a cache of its own


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "6 heads for 4"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "lacks 'conv'"),
    (lambda c: c["layers"][1]["mixer"].pop("diff"), "lacks 'diff'"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("fast"), "lacks 'fast'"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=10), "takes 10 of 6 experts and 3"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda c: c["layers"][3]["mlp"].update(kind="wide"), "unknown kind"),
    (lambda c: c["loop"].update(stop=9), "loop runs layers"),
    (lambda c: c["loop"].update(times=0), "0 times"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_config_errors_name_the_place(edit, text):
    raw = json.loads(json.dumps(CONFIGS["K"]))
    edit(raw)
    with pytest.raises(ConfigError, match=text):
        get_architecture("Ferodra").load_config(raw)


def test_tensor_names_and_cache_needs(tmp_path):
    arch = get_architecture("Ferodra")
    names = declare_tensors(arch, arch.build_spec(arch.load_config(CONFIGS["K"])))
    for n in ("embed", "loop.step", "final.norm", "final.norm.alpha", "final.norm.b", "l0.norm1", "l0.norm1.alpha", "l0.norm1b.b", "l0.norm2",
              "l0.norm2b.alpha", "l0.ls1", "l0.ls2", "l0.mix.q", "l0.mix.q.conv", "l0.mix.b", "l0.mix.a", "l0.mix.A_log", "l0.mix.dt_bias",
              "l0.mix.g", "l0.mix.norm", "l0.mlp.router", "l0.mlp.correction", "l0.mlp.e4.up", "l0.mlp.shared.down", "l0.mlp.shared.sg",
              "l1.mix.lq1", "l1.mix.lk2", "l1.ls1", "l3.mlp.gate", "l3.mlp.down"):
        assert n in names, n
    for n in ("head", "l1.norm2", "l1.norm2b", "l1.ls2", "l1.mlp.router", "l2.mlp.shared.up", "l2.mlp.shared.sg", "l0.mlp.e5.up", "l0.mlp.e0.gate",
              "l0.mix.a1", "l0.mix.g1", "l3.mlp.router"):
        assert n not in names, n
    assert names["loop.step"].shape == (2, 96) and names["l0.norm1.alpha"].shape == () and names["l0.mix.dt_bias"].shape == (6,)
    assert names["l0.mix.a"].shape == (6, 96) and names["l0.mix.g"].shape == (240, 96) and names["l0.mix.v.conv"].shape == (240, 4)
    assert names["l1.mix.q"].shape == (6 * 2 * 16, 96) and names["l1.mix.k"].shape == (2 * 2 * 16, 96) and names["l1.mix.o"].shape == (96, 144)
    assert names["l2.mlp.router"].shape == (9, 96) and names["l2.mlp.correction"].shape == (9,) and names["l0.mlp.shared.sg"].shape == (1, 96)
    d = write_case(tmp_path, "K", store_dtype=torch.float32)
    with ops.use_kernels(FakeKernels()):
        needs = Model.from_folder(d, "float32", "cpu").cache_needs()
    # run order 0 | 1 2 | 1 2 | 3: caches 0 .. 5
    assert sorted(needs) == [0, 1, 2, 3, 4, 5]
    assert needs[1] == needs[3] == KVNeed(2, 32, None, 24) and needs[2] == needs[4] == KVNeed(4, 48, None, 16)
    assert needs[0] == StateNeed((6 * 40 * 24 + 3 * (2 * 48 + 240),), torch.float32)


# ---- the host side under every way of cutting the work -------------------------------------------------
@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    root = tmp_path_factory.mktemp("ferodra")
    out = {}
    for name in CONFIGS:
        d = write_case(root, name, store_dtype=torch.float32)
        with ops.use_kernels(FakeKernels()):
            out[name] = (d, Model.from_folder(d, "float32", "cpu"))
    return out


LENGTHS = {"K": [1, 9, 40, 75], "L": [3, 35, 50, 20, 2], "M": [2, 70, 33], "N": [45, 5, 20], "R": [41, 3, 30]}


def test_the_stream_after_every_layer_run(cases):
    """The residual stream the engine holds after each layer run is the plain implementation's (the addend a layer still owes
    is added here by hand; the vector of the next run is not part of it)."""
    for name, vocab in (("K", 211), ("L", 300)):
        d, model = cases[name]
        toks = random_tokens(vocab, 12, 3)
        cfg, w = plain.load_folder(d)
        _, streams = plain.forward(cfg, w, toks, return_layers=True)
        seen = []

        def spy(fn):
            def run(residual, delta, ctx, cache, writes_cache, select_rows):
                res, d_ = fn(residual, delta, ctx, cache, writes_cache, select_rows)      # every row is wanted: nothing is gathered
                seen.append(res.double() + owed(d_))
                return res, d_
            return run
        try:
            for b in model.blocks:
                b.forward = spy(b.forward)
            with ops.use_kernels(FakeKernels()):
                rp = TraceReplayer(model, 64, 16, 2, native=False)
                rp.run_step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": list(range(12))}], "end": ["a"]})
        finally:
            for b in model.blocks:
                del b.forward
        assert len(seen) == streams.shape[0] == len(plain.run_order(cfg))
        for i, x in enumerate(seen):
            assert (x - streams[i]).abs().max() < 1e-4, f"{name}: layer run {i}"


def test_every_run_gets_a_vector_of_its_own(cases):
    """Swapping the vectors of two runs changes the logits: the run order's number picks the row."""
    d, _ = cases["L"]
    cfg, w = plain.load_folder(d)
    toks = random_tokens(300, 9, 4)
    base = plain.forward(cfg, w, toks)
    w2 = dict(w, **{"loop.step": w["loop.step"][[1, 0, 2]]})
    assert (plain.forward(cfg, w2, toks) - base).abs().max() > 1e-3


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_replay_matches_plain_under_every_cut(cases, name):
    d, model = cases[name]
    reqs = {f"r{i}": random_tokens(CONFIGS[name]["vocab"], n, 40 + i) for i, n in enumerate(LENGTHS[name])}
    want = plain_logits(d, reqs)
    rounded = max(-(-len(t) // 64) * 64 for t in reqs.values())
    for what, steps, cap in (("whole", trace_whole(reqs), rounded), ("tail", trace_tail(reqs, 20), rounded),
                             ("portions", trace_portions(reqs), rounded), ("mixed", trace_mixed(reqs, 2 * rounded, seed=3), 2 * rounded)):
        with ops.use_kernels(FakeKernels()):
            rp = TraceReplayer(model, cap, BLOCK_SIZE[name], 4, native=False)
            got = replay_and_collect(rp, steps)
        rp.runner.manager.check_invariants()
        assert all(p.num_free == p.num_blocks for p in rp.runner.manager.pools), "pages were lost"
        assert len(got) == sum(len(t) for t in reqs.values())
        bad = first_bad(got, want, 3e-4)
        assert bad is None, f"{name} {what}: first wrong logits at {bad}; worst {max_error(got, want)}"


def test_a_slot_that_is_used_again_starts_from_zero(cases):
    """Two state slots, five requests one after another and side by side: a request that inherits a slot must not see what the
    one before left in the matrix or in the convolution's tail."""
    d, model = cases["K"]
    reqs = {f"r{i}": random_tokens(211, n, 90 + i) for i, n in enumerate([30, 12, 25, 7, 18])}
    want = plain_logits(d, reqs)
    steps = trace_mixed(reqs, 128, seed=1, max_live=2)
    with ops.use_kernels(FakeKernels()):
        rp = TraceReplayer(model, 128, 16, 2, native=False)
        got = replay_and_collect(rp, steps)
    bad = first_bad(got, want, 3e-4)
    assert bad is None, f"first wrong logits at {bad}"


def test_greedy_generation_through_the_scheduler(cases):
    d, model = cases["L"]
    cfg, w = plain.load_folder(d)
    prompts = [random_tokens(300, n, 70 + i) for i, n in enumerate([1, 6, 30, 50])]

    def greedy(prompt, n):
        toks = list(prompt)
        for _ in range(n):
            toks.append(int(torch.argmax(plain.forward(cfg, w, toks)[-1])))
        return toks[len(prompt):]
    want = [greedy(p, 4) for p in prompts]
    for kw in (dict(budget=64, kv_cache_tokens=512), dict(budget=11, kv_cache_tokens=512),        # whole prompts; portions
               dict(budget=16, kv_cache_tokens=96, enable_prefix_caching=True)):                   # few pages: preemption
        sched = SchedulerConfig(max_num_batched_tokens=kw.pop("budget"), max_num_seqs=4)
        with ops.use_kernels(FakeKernels()):
            eng = Engine(model, EngineConfig(dtype="float32", block_size=8, warmup=False, sched=sched, max_model_len=96, **kw))
            assert not eng.runner.prefix_caching                   # a model with state cannot start behind a shared prefix
            assert eng.generate(prompts, max_tokens=4, temperature=0.0) == want
        eng.cache.check_invariants()
        assert all(p.num_free == p.num_blocks for p in eng.cache.pools)


def test_command_line_writes_and_loads_a_folder(tmp_path):
    """``iian random-weights`` from a Ferodra config.json, then the folder through the loader (names, shapes, the plug-in)."""
    from iian_b200.cli.main import main as cli_main
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(CONFIGS["M"]))
    out = tmp_path / "model"
    assert cli_main(["random-weights", str(cfg_path), str(out), "--seed", "3"]) == 0
    arch, cfg = load_model_config(str(out))
    assert arch.name == "Ferodra" and cfg == arch.load_config(CONFIGS["M"])
    with ops.use_kernels(FakeKernels()):
        model = Model.from_folder(str(out), "float32", "cpu")
        rp = TraceReplayer(model, 64, 16, 2, native=False)
        logits = rp.run_step({"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [2]}], "end": ["a"]})
    want = plain.forward(*plain.load_folder(str(out)), [1, 2, 3])[-1]
    assert (logits[0].double() - want).abs().max() < 3e-4
