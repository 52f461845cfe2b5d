"""Tatelorn without a GPU: the plain implementation's mechanisms on cases worked out by hand, the configuration reader, the tensor
names, and the engine's host side (a stream that starts with a row per position and a norm, sub-layers that read the stream itself,
values that take a share of the first mixing layer's, page reuse, portions, mixed batches, the scheduler's entry point) with the
torch stand-in for the kernels against the plain implementation."""
import json
import math

import pytest
import torch

from helpers import first_bad, max_error, random_tokens, replay_and_collect, trace_mixed, trace_portions, trace_tail, trace_whole
import plain_tatelorn as plain
from fake_kernels import FakeKernels
from iian_b200 import EngineConfig, SchedulerConfig, ops
from iian_b200.config.registry import get_architecture, load_model_config
from iian_b200.engine.engine import Engine
from iian_b200.engine.model import Model, declare_tensors
from iian_b200.engine.replay import TraceReplayer
from iian_b200.models.qwen3 import ConfigError
from iian_b200.parts.base import KVNeed
from tatelorn_cases import BLOCK_SIZE, CONFIGS, owed, plain_logits, write_case

F64 = torch.float64


def t64(*v):
    return torch.tensor(v, dtype=F64)


# ---- the plain implementation's mechanisms ------------------------------------------------------------
def test_plain_norm_weight_sits_around_zero():
    got = plain.centred_norm(t64(3.0, -4.0)[None], t64(0.0, 0.5), 0.0)
    r = math.sqrt(12.5)
    assert torch.allclose(got, t64(3 / r, -6 / r)[None])
    assert torch.allclose(plain.centred_norm(t64(0.0, 0.0)[None], t64(1.0, 1.0), 1e-6), t64(0.0, 0.0)[None])
    assert torch.allclose(plain.centred_norm(t64(1.0, 1.0)[None], t64(0.0, 0.0), 3.0), t64(0.5, 0.5)[None])      # eps inside the root


def test_plain_embedding_scales_the_token_and_not_the_position():
    w = {"embed": t64(1.0, 0.0, 0.0, 2.0).view(2, 2), "pos": t64(0.0, 0.0, 5.0, 0.0).view(2, 2), "embed.norm": t64(0.0, 1.0)}
    got = plain.placed_embedding(w, [1, 0], 3.0, 0.0)
    r = math.sqrt(32.0)                                    # the second row: 3 * (1, 0) + (5, 0)
    assert torch.allclose(got, t64(0.0, 2 * 6 / math.sqrt(18.0), 8 / r, 0.0).view(2, 2))


def test_plain_head_has_one_more_in_the_denominator():
    q, k, v = t64(2.0).view(1, 1), t64(1.0, -1.0).view(2, 1), t64(10.0, 20.0).view(2, 1)
    # position 0 sees key 0 alone: e^2 / (1 + e^2) of its value, not all of it
    got = plain.capped_softmax_head(q, k, v, 1.0, None)
    assert got.item() == pytest.approx(10 * math.exp(2) / (1 + math.exp(2)))
    got = plain.capped_softmax_head(q, k, v, 0.5, None, q_pos0=1)
    a, b = math.exp(1.0), math.exp(-1.0)
    assert got.item() == pytest.approx((10 * a + 20 * b) / (1 + a + b))
    # scores far below the extra term's 0 leave almost nothing, scores far above it everything
    low = plain.capped_softmax_head(q, -20 * torch.ones_like(k), v, 1.0, None, q_pos0=1)
    high = plain.capped_softmax_head(q, 20 * torch.ones_like(k), v, 1.0, None, q_pos0=1)
    assert abs(low.item()) < 1e-14 and high.item() == pytest.approx(15.0)


def test_plain_cap_bends_scores_and_keeps_them_below_it():
    q, k, v = t64(1.0).view(1, 1), t64(1.0, 30.0).view(2, 1), t64(1.0, 2.0).view(2, 1)
    a, b = math.exp(2 * math.tanh(0.5)), math.exp(2 * math.tanh(15.0))
    got = plain.capped_softmax_head(q, k, v, 1.0, 2.0, q_pos0=1)
    assert got.item() == pytest.approx((a + 2 * b) / (1 + a + b))


def test_plain_mixed_values_and_groups():
    v, f = t64(4.0, 0.0), t64(0.0, 8.0)
    assert torch.equal(plain.mixed_values(v, None, 0.25), v)
    assert torch.allclose(plain.mixed_values(v, f, 0.25), t64(3.0, 2.0))
    # heads 0, 1 read key/value head 0, heads 2, 3 head 1
    k = torch.zeros(1, 2, 3, dtype=F64)
    out = plain.grouped_attention(torch.zeros(1, 4, 3, dtype=F64), k, t64(2.0, 6.0).view(1, 2, 1), 1.0, 5.0)
    assert out.view(4).tolist() == [1.0, 1.0, 3.0, 3.0]               # score 0 against the extra term's 0: half each


def test_the_first_mixing_layer_gives_its_own_values():
    """A layer that does not mix neither gives nor takes; the first that mixes ignores its own number."""
    cfg = CONFIGS["K"]
    g = torch.Generator().manual_seed(5)
    arch = get_architecture("Tatelorn")
    w = {n: torch.randn(ts.shape, generator=g, dtype=F64) * 0.2 for n, ts in
         declare_tensors(arch, arch.build_spec(arch.load_config(cfg))).items()}
    assert "l1.mix.vmix" in w and "l3.mix.vmix" in w and "l0.mix.vmix" not in w and "l2.mix.vmix" not in w
    toks = random_tokens(211, 7, 6)
    base = plain.forward(cfg, w, toks)
    assert torch.equal(plain.forward(cfg, dict(w, **{"l1.mix.vmix": w["l1.mix.vmix"] + 1}), toks), base)
    assert (plain.forward(cfg, dict(w, **{"l3.mix.vmix": w["l3.mix.vmix"] + 1}), toks) - base).abs().max() > 1e-3
    # with a share of 1 the last layer uses layer 1's values alone: its own value matrix has no say
    w1 = dict(w, **{"l3.mix.vmix": torch.ones((), dtype=F64)})
    assert torch.equal(plain.forward(cfg, dict(w1, **{"l3.mix.v": -w["l3.mix.v"]}), toks), plain.forward(cfg, w1, toks))
    assert (plain.forward(cfg, dict(w1, **{"l1.mix.v": -w["l1.mix.v"]}), toks) - plain.forward(cfg, w1, toks)).abs().max() > 1e-3


def test_plain_feed_forwards():
    w = {"gate": t64(1.0, -1.0).view(2, 1), "up": t64(2.0, 3.0).view(2, 1), "down": t64(1.0, 10.0).view(1, 2)}
    assert plain.relu_feed_forward(t64(2.0).view(1, 1), w, "").item() == pytest.approx(2 * 4.0)              # the second gate is shut
    h = t64(2.0).view(1, 1)
    g0, u0, g1, u1 = 1.5, 1.5, -2.0, 1.5                   # clipped: gate above only, up on both sides
    want = g0 / (1 + math.exp(-1.702 * g0)) * (u0 + 1) + 10 * g1 / (1 + math.exp(-1.702 * g1)) * (u1 + 1)
    assert plain.clipped_expert(h, w, "", 1.5).item() == pytest.approx(want)
    low = plain.clipped_expert(h, dict(w, up=t64(-4.0, 0.0).view(2, 1)), "", 1.5).item()
    assert low == pytest.approx(g0 / (1 + math.exp(-1.702 * g0)) * (1 - 1.5) + 10 * g1 / (1 + math.exp(-1.702 * g1)))


def test_plain_router_weighs_the_chosen_ones_only():
    w = {"router": t64(1.0, 3.0, 2.0, 3.0).view(4, 1)}
    ids, wts = plain.router_choice(t64(1.0).view(1, 1), w, "", 3)
    assert ids.tolist() == [[1, 3, 2]]                                 # a tie goes to the lower index
    e = [math.exp(3), math.exp(3), math.exp(2)]
    assert wts[0].tolist() == pytest.approx([x / sum(e) for x in e])


# ---- configuration, names, what the caches must hold ------------------------------------------------------
def test_config_round_trip_and_spec():
    arch = get_architecture("Tatelorn")
    for name, raw in CONFIGS.items():
        c = arch.load_config(raw)
        assert arch.load_config(arch.config_to_dict(c)) == c, name
        spec = arch.build_spec(c)
        spec.validate()
        assert spec.max_position == raw["max_positions"]
        assert [ls.mixer["value_mix"] for ls in spec.layers] == {
            "K": [None, "first", None, "later"], "L": ["first", "later", "later"], "M": [None, None],
            "N": ["first", None, "later", "later"], "R": ["first", "later", "later"]}[name]


def test_config_takes_the_number_of_positions_from_the_table(tmp_path):
    d = write_case(tmp_path, "M", store_dtype=torch.float32)
    raw = json.loads((tmp_path / d.split("/")[-1] / "config.json").read_text())
    raw.pop("max_positions")
    (tmp_path / d.split("/")[-1] / "config.json").write_text(json.dumps(raw))
    _, cfg = load_model_config(d)
    assert cfg.max_positions == 300


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "6 heads for 4"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "lacks 'scale'"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"].update(v_mix=1), "v_mix"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=20), "layer 1, which have other sizes"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "takes 6 of 5"),
    (lambda c: c["layers"][1]["mlp"]["expert"].update(limit=0), "limit"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("limit"), "lacks 'limit'"),
    (lambda c: c["layers"][3]["mlp"].update(kind="wide"), "unknown kind"),
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_config_errors_name_the_place(edit, text):
    raw = json.loads(json.dumps(CONFIGS["K"]))
    edit(raw)
    with pytest.raises(ConfigError, match=text):
        get_architecture("Tatelorn").load_config(raw)


def test_tensor_names_and_cache_needs(tmp_path):
    arch = get_architecture("Tatelorn")
    names = declare_tensors(arch, arch.build_spec(arch.load_config(CONFIGS["K"])))
    for n in ("embed", "pos", "embed.norm", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.q", "l0.mix.k.norm", "l0.mix.o", "l0.mlp.gate",
              "l1.mix.vmix", "l1.mlp.router", "l1.mlp.e4.up", "l1.mlp.shared.gate", "l1.mlp.shared.sg", "l2.norm1", "l3.mix.vmix",
              "l3.mlp.e5.down"):
        assert n in names, n
    for n in ("head", "l0.norm1b", "l2.norm2", "l0.mix.vmix", "l2.mix.vmix", "l2.mlp.gate", "l1.mlp.router.b", "l1.mlp.e5.up",
              "l3.mlp.shared.sg", "l0.mix.sink"):
        assert n not in names, n
    assert names["pos"].shape == (400, 96) and names["l1.mix.vmix"].shape == () and names["l1.mix.q.norm"].shape == (16,)
    assert names["l1.mix.v"].shape == (48, 96) and names["l1.mix.o"].shape == (96, 144) and names["l1.mlp.shared.sg"].shape == (1, 96)
    d = write_case(tmp_path, "K", store_dtype=torch.float32)
    with ops.use_kernels(FakeKernels()):
        needs = Model.from_folder(d, "float32", "cpu").cache_needs()
    assert needs == {0: KVNeed(2, 24, None, 40), 1: KVNeed(2, 16, None, 24), 2: KVNeed(3, 20, None, 12), 3: KVNeed(2, 28, None, 24)}


# ---- the host side under every way of cutting the work -------------------------------------------------
@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    root = tmp_path_factory.mktemp("tatelorn")
    out = {}
    for name in CONFIGS:
        d = write_case(root, name, store_dtype=torch.float32)
        with ops.use_kernels(FakeKernels()):
            out[name] = (d, Model.from_folder(d, "float32", "cpu"))
    return out


LENGTHS = {"K": [1, 9, 40, 75], "L": [3, 35, 50, 20, 2], "M": [2, 70, 33], "N": [45, 5, 20], "R": [41, 3, 30]}


def test_the_stream_after_every_layer(cases):
    """The residual stream the engine holds after each layer is the plain implementation's (the addend a layer still owes is
    added here by hand)."""
    for name in ("K", "L", "R"):
        d, model = cases[name]
        toks = random_tokens(CONFIGS[name]["vocab"], 12, 3)
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
        assert len(seen) == streams.shape[0]
        for i, x in enumerate(seen):
            assert (x - streams[i]).abs().max() < 1e-4, f"{name}: layer {i}"


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


def test_a_bfloat16_model_runs_through_the_stand_ins(cases, tmp_path):
    """The path with a 16-bit copy of the stream (the embedding's for the first layer, the identity norm's behind it) gives what
    rounding allows."""
    d = write_case(tmp_path, "L", steady=True)
    with ops.use_kernels(FakeKernels()):
        model = Model.from_folder(d, "bfloat16", "cpu")
        reqs = {"a": random_tokens(300, 21, 1)}
        got = replay_and_collect(TraceReplayer(model, 64, 8, 2, native=False), trace_portions(reqs))
    want = plain_logits(d, reqs)
    scale = (want["a"] - want["a"].mean(-1, keepdim=True)).pow(2).mean().sqrt().item()
    worst, where = max_error(got, want)
    assert worst < 0.3 * scale, (worst, scale, where)


def test_a_request_beyond_the_position_table_is_refused(cases):
    d, model = cases["R"]
    with ops.use_kernels(FakeKernels()):
        eng = Engine(model, EngineConfig(dtype="float32", block_size=16, warmup=False, kv_cache_tokens=512,
                                         sched=SchedulerConfig(max_num_batched_tokens=64, max_num_seqs=2)))
        assert eng.generate([random_tokens(150, 280, 1)], max_tokens=10, temperature=0.0)[0]
        with pytest.raises(ValueError):
            eng.generate([random_tokens(150, 291, 1)], max_tokens=1, temperature=0.0)


def test_greedy_generation_through_the_scheduler(cases):
    d, model = cases["L"]
    cfg, w = plain.load_folder(d)
    prompts = [random_tokens(300, n, 70 + i) for i, n in enumerate([1, 6, 30, 50])]
    prompts.append(prompts[3][:40] + [7, 9])                           # shares two pages of five with another

    def greedy(prompt, n):
        toks = list(prompt)
        for _ in range(n):
            toks.append(int(torch.argmax(plain.forward(cfg, w, toks)[-1])))
        return toks[len(prompt):]
    want = [greedy(p, 4) for p in prompts]
    for kw in (dict(budget=64, kv_cache_tokens=512), dict(budget=11, kv_cache_tokens=512),        # whole prompts; portions
               dict(budget=16, kv_cache_tokens=96),                                                # few pages: preemption
               dict(budget=64, kv_cache_tokens=512, enable_prefix_caching=True)):                  # cached values are the mixed ones
        sched = SchedulerConfig(max_num_batched_tokens=kw.pop("budget"), max_num_seqs=4)
        with ops.use_kernels(FakeKernels()):
            eng = Engine(model, EngineConfig(dtype="float32", block_size=8, warmup=False, sched=sched, max_model_len=96, **kw))
            assert eng.generate(prompts, max_tokens=4, temperature=0.0) == want
            if kw.get("enable_prefix_caching"):
                assert eng.runner.prefix_caching
                assert eng.generate(prompts, max_tokens=4, temperature=0.0) == want                # everything behind a known prefix
        eng.cache.check_invariants()


def test_command_line_writes_and_loads_a_folder(tmp_path):
    """``iian random-weights`` from a Tatelorn config.json, then the folder through the loader (names, shapes, the plug-in)."""
    from iian_b200.cli.main import main as cli_main
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(CONFIGS["M"]))
    out = tmp_path / "model"
    assert cli_main(["random-weights", str(cfg_path), str(out), "--seed", "3"]) == 0
    arch, cfg = load_model_config(str(out))
    assert arch.name == "Tatelorn" and cfg == arch.load_config(CONFIGS["M"])
    with ops.use_kernels(FakeKernels()):
        model = Model.from_folder(str(out), "float32", "cpu")
        rp = TraceReplayer(model, 64, 16, 2, native=False)
        logits = rp.run_step({"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [2]}], "end": ["a"]})
    want = plain.forward(*plain.load_folder(str(out)), [1, 2, 3])[-1]
    assert (logits[0].double() - want).abs().max() < 3e-4
