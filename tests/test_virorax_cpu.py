"""Virorax without a GPU: the configuration reader and what it refuses, the model as the registry builds it (a loop's runs with
caches and states of their own), the plain implementation's own checks (each mechanism against its sum written out or on
made-up inputs), and the engine around the kernels (cache pages, state slots, step function, scheduler) under every way of
cutting the work, with the kernels replaced by their torch statements."""
import copy
import json
import math
import os

import pytest
import torch

import plain_virorax as plain
import traces
from arle_b200 import Engine
from arle_b200.config import ConfigError, ViroraxConfig, config_from_dict, load_config
from arle_b200.engine import ModelRunner, StepEntry, load_model
from arle_b200.parts import build_model, build_part
from arle_b200.parts.attention import AttentionSpec
from arle_b200.parts.block import OutputNormBlockSpec
from arle_b200.parts.lightning import ConstantDecayAttentionSpec
from arle_b200.parts.norm import RmsNormSpec
from arle_b200.parts.rotary import RotarySpec
from arle_b200.sampling import SamplingParams
from tiny_virorax import CONFIGS, PAGE_SIZES, make_model_dir, read_model

LENGTHS = {"V1": [1, 5, 12, 23, 70, 33], "V2": [2, 17, 40, 64, 9, 31], "R": [3, 30, 11, 2, 45], "L": [1, 20, 33, 7], "S": [3, 30, 11, 2, 45]}
F64 = torch.float64
_cache = {}


def model_and_oracle(name, tmp_path_factory):
    if name not in _cache:
        d = make_model_dir(name, seed=21, root=str(tmp_path_factory.mktemp(f"tiny{name}")))
        cfg, w = read_model(d)
        reqs = traces.make_requests(cfg["vocab"], LENGTHS[name], seed=6)
        _cache[name] = (d, cfg, w, reqs, {r: plain.forward(cfg, w, t) for r, t in reqs.items()})
    return _cache[name]


# ------------------------------------------------------------------ configuration
def test_registry_finds_the_architecture_and_reads_every_size():
    cfg = config_from_dict(CONFIGS["V1"])
    assert isinstance(cfg, ViroraxConfig) and [l.type for l in cfg.layers] == ["attention", "retention", "attention", "retention"]
    a, r = cfg.layers[:2]
    assert (a.m("window"), a.m("vdim"), a.m("rot_dims"), a.m("rot_base"), a.m("scale"), a.ff) == (7, 24, 8, 10000.0, 0.3, 40)
    assert (r.m("decay"), r.m("dim"), r.m("vdim"), r.m("rot_dims"), r.ff) == ((0.6, 0.9, 0.999), 8, 12, 4, 0)
    assert (cfg.norm_eps, cfg.residual_mult, cfg.logit_softcap, cfg.max_positions) == (1e-5, 0.45, 9.0, 512)
    assert (cfg.loop.start, cfg.loop.stop, cfg.loop.times) == (1, 3, 2)
    v2 = config_from_dict(CONFIGS["V2"])
    assert v2.logit_softcap is None and v2.layers[2].m("window") is None and v2.layers[0].m("rot_dims") == 0
    assert config_from_dict(CONFIGS["A"]).loop is None


def test_model_spec_runs_the_loop_with_caches_and_states_of_its_own():
    spec = config_from_dict(CONFIGS["V1"]).to_model_spec()
    assert [(e.block, e.add_embedding) for e in spec.schedule] == [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)]
    assert all(e.keys_of is None for e in spec.schedule)
    model = build_model(spec)
    assert model.entry_cache_layer == [0, None, 1, None, 2, None] and model.entry_state == [None, 0, None, 1, None, 2]
    assert model.cache_needs[0].arrays() == ((2, 16), (2, 24)) and [n.window for n in model.cache_needs] == [7, 11, 11]
    assert [n.shape for n in model.state_needs] == [(3 * 8 * 12,), (3 * 8 * 12,), (2 * 16 * 8,)]
    decls = {d.name: d.shape for d in model.weight_decls()}
    assert decls["pos"] == (512, 64) and decls["l0.mix.q.b"] == (64,) and decls["l0.mix.v.b"] == (48,) and decls["l0.mix.sink"] == (4,)
    assert decls["l0.mix.g"] == (4, 64) and decls["l0.mix.q.norm"] == (16,) and decls["l1.mix.g"] == (36, 64) and decls["l0.mlp.up"] == (40, 64)
    assert not {"l0.mix.o.b", "l1.mix.norm", "l1.norm2", "head", "l1.mix.q.b", "l1.mlp.up"} & set(decls)
    v2 = config_from_dict(CONFIGS["V2"]).to_model_spec()
    assert [e.block for e in v2.schedule] == [0, 1, 2, 3] * 3 and [e.add_embedding for e in v2.schedule] == [i in (4, 8) for i in range(12)]
    once = dict(CONFIGS["V1"], loop={"start": 1, "stop": 3, "times": 1})
    assert [(e.block, e.add_embedding) for e in config_from_dict(once).to_model_spec().schedule] == [(i, False) for i in range(4)]
    v3 = config_from_dict(CONFIGS["V3"]).to_model_spec()
    assert [(e.block, e.add_embedding) for e in v3.schedule][3:] == [(3, False), (4, False), (3, True), (4, False)]       # to the last layer


def test_rows_of_the_position_table_stand_in_for_a_missing_key(tmp_path):
    d = make_model_dir("A", root=str(tmp_path))
    cfg = {k: v for k, v in CONFIGS["A"].items() if k != "max_positions"}
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    assert load_config(d).max_positions == 512
    with pytest.raises(ConfigError, match="max_positions"):
        config_from_dict(cfg)


@pytest.mark.parametrize("change,match", [
    (lambda c: c["layers"][0].update(type="wkv"), "type"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=0.0), "rot.base"),
    (lambda c: c["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=300), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mixer"].update(heads=3), "heads"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.5, -0.1]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(dim=600), "dim"),
    (lambda c: c["layers"][0].update(mlp={"kind": "moe", "ff": 8}), "mlp"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["loop"].pop("times"), "times"),
    (lambda c: c.update(logit_softcap=0.0), "logit_softcap"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c["norm"].update(eps=0.0), "norm.eps"),
])
def test_configuration_errors_name_the_key(change, match):
    c = copy.deepcopy(CONFIGS["V1"])
    change(c)
    with pytest.raises(ConfigError, match=match):
        config_from_dict(c)


def test_parts_refuse_what_their_kernels_do_not_do():
    rot = RotarySpec(8, 100.0)
    with pytest.raises(ValueError):              # a rotation of more numbers than a head has
        build_part(ConstantDecayAttentionSpec("m.", 32, 2, 4, 8, (0.5, 0.5), 1e-5, activation="none", position=rot))
    with pytest.raises(ValueError):              # a rotation behind an activation
        build_part(ConstantDecayAttentionSpec("m.", 32, 2, 8, 8, (0.5, 0.5), 1e-5, position=rot))
    with pytest.raises(ValueError):
        build_part(ConstantDecayAttentionSpec("m.", 32, 2, 8, 8, (0.5, 0.5), 1e-5, norm="rows"))
    with pytest.raises(ValueError):              # stored sinks and a constant one
        build_part(AttentionSpec("m.", 32, 2, 1, 8, 0.3, 1e-5, rot, stored_sinks=True, sink=0.0))
    spec = config_from_dict(CONFIGS["A"]).to_model_spec()
    block = OutputNormBlockSpec(mixer_norm=RmsNormSpec("n", 64, 1e-5), mixer=spec.blocks[0].mixer)
    with pytest.raises(ValueError, match="factor"):         # a branch that is normed on its way into the residual has no factor
        build_model(type(spec)(**{**spec.__dict__, "blocks": (block,)}))


# ------------------------------------------------------------ the plain implementation
def _rand(g, *shape):
    return torch.randn(*shape, generator=g, dtype=F64)


def test_plain_memory_equals_its_sum_written_out():
    """o_t = sum_(s <= t) decay^(t - s) (q_t . k_s) v_s per head."""
    g = torch.Generator().manual_seed(0)
    T, H, D, Dv = 9, 3, 5, 4
    q, k, v = _rand(g, T, H, D), _rand(g, T, H, D), _rand(g, T, H, Dv)
    decay = [0.0, 0.93, 1.0]
    got = plain.decaying_memory(q, k, v, decay)
    for h in range(H):
        for t in range(T):
            want = sum(decay[h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1))
            assert torch.allclose(got[t, h], want, atol=1e-12)


def test_plain_sinks_window_rotation_cap_and_norm_on_made_up_inputs():
    g = torch.Generator().manual_seed(1)
    see = plain.within_window(12, 4)
    assert see[9].nonzero().flatten().tolist() == [6, 7, 8, 9] and see[2].nonzero().flatten().tolist() == [0, 1, 2]
    assert plain.within_window(5)[4].all() and not plain.within_window(5)[2, 3]
    # weights written out: e^s / (e^sink + sum e^s), a sink of its own per head, key heads shared by groups of query heads
    q, k, v = _rand(g, 5, 4, 6), _rand(g, 5, 2, 6), _rand(g, 5, 2, 3)
    sinks = torch.tensor([-3.0, 0.5, 2.0, 8.0], dtype=F64)
    got = plain.sink_attention(q, k, v, 0.7, plain.within_window(5, 3), sinks)
    for h in range(4):
        e = [math.exp(0.7 * float(q[4, h] @ k[j, h // 2])) for j in (2, 3, 4)]
        want = sum(e[n] * v[j, h // 2] for n, j in enumerate((2, 3, 4))) / (math.exp(float(sinks[h])) + sum(e))
        assert torch.allclose(got[4, h], want)
    far = torch.full((4,), -200.0, dtype=F64)
    assert torch.allclose(plain.sink_attention(q, k, v, 0.7, plain.within_window(5), far), plain.sink_attention(q, k, v, 0.7, plain.within_window(5), None))
    x = _rand(g, 5, 2, 8)
    r = plain.rotate_halves(x, torch.arange(5), 100.0, 4)
    assert torch.equal(r[..., 4:], x[..., 4:]) and torch.allclose(r[0], x[0])
    a = 3 * 100.0 ** (-2 * 1 / 4)
    assert torch.allclose(r[3, 1, 1], x[3, 1, 1] * math.cos(a) - x[3, 1, 3] * math.sin(a))
    assert torch.allclose(r[3, 1, 3], x[3, 1, 3] * math.cos(a) + x[3, 1, 1] * math.sin(a))
    z = torch.tensor([-100.0, 0.0, 0.1, 5.0, 1e6], dtype=F64)
    c = plain.capped(z, 5.0)
    assert abs(float(c[3]) - 5.0 * math.tanh(1.0)) < 1e-12 and float(c.abs().max()) <= 5.0 and abs(float(c[2]) - 0.1) < 1e-4
    u = plain.unit_rms(3.0 * x, 0.0)
    assert torch.allclose((u * u).mean(-1), torch.ones(5, 2, dtype=F64)) and torch.allclose(u, plain.unit_rms(x, 0.0))


def test_plain_loop_order_and_causality(tmp_path):
    assert plain.runs({"layers": [0] * 4}) == [(i, False) for i in range(4)]
    assert plain.runs({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 3}}) == [
        (0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    d = make_model_dir("V1", seed=5, root=str(tmp_path))
    cfg, w = read_model(d)
    toks = traces.make_requests(cfg["vocab"], [30], seed=1)["r0"]
    base = plain.forward(cfg, w, toks)
    assert (plain.forward(cfg, w, toks[:17]) - base[:17]).abs().max() < 1e-12
    # two passes of a loop are the layers written out twice, with the embedding output added between them
    flat = copy.deepcopy(cfg)
    flat.pop("loop")
    flat["layers"] = [cfg["layers"][i] for i in (0, 1, 2, 1, 2, 3)]
    names = {}
    for n, i in enumerate((0, 1, 2, 1, 2, 3)):
        names.update({f"l{n}." + t[len(f"l{i}."):]: w[t] for t in w if t.startswith(f"l{i}.")})
    unrolled = {**{t: w[t] for t in ("embed", "pos", "final.norm")}, **names}
    assert (plain.forward(flat, unrolled, toks) - base).abs().max() > 1e-3         # without the added embedding output: another model
    lo = []
    plain.forward(cfg, w, toks, layers_out=lo)
    assert len(lo) == 6


# ------------------------------------------------------------------ the engine on the CPU
@pytest.mark.parametrize("cut", ["whole", "tail_decode", "portions", "mixed"])
@pytest.mark.parametrize("name", ["V1", "V2", "R", "L"])
def test_cuttings_cpu(name, cut, tmp_path_factory, cpu_kernels):
    d, cfg, w, reqs, oracle = model_and_oracle(name, tmp_path_factory)
    steps = traces.mixed(reqs, seed=4) if cut == "mixed" else getattr(traces, cut)(reqs)
    ps = PAGE_SIZES[name]
    runner = ModelRunner(load_model(d, torch.float32, "cpu"), ps, max(1, traces.peak_tokens(steps) // ps), 4, device="cpu")
    got = traces.run_trace(runner, steps)
    runner.cache.check()
    assert runner.cache.num_free_slots == 4 and all(g.pool.num_free == g.pool.num_pages for g in runner.cache.groups)
    for r, want in oracle.items():
        err = (got[r].double() - want).abs().max().item()
        assert err < 5e-4 * float(want.std()), f"{name} {cut}: request {r}, error {err:.3g}"


def test_window_pages_go_back_while_the_request_lives(tmp_path_factory, cpu_kernels):
    d, cfg, w, reqs, oracle = model_and_oracle("V1", tmp_path_factory)
    runner = ModelRunner(load_model(d, torch.float32, "cpu"), 4, 40, 2, device="cpu")
    toks = reqs["r4"]
    runner.step([StepEntry("a", toks[:50], ())])
    # token 50 sees from 44 on (window 7) and from 40 on (window 11, of both passes): pages 11, 12 and 10, 11, 12
    assert [g.pool.num_pages - g.pool.num_free for g in runner.cache.groups] == [2, 3]
    lg = runner.step([StepEntry("a", toks[50:], range(20))])
    assert (lg.double() - oracle["r4"][50:]).abs().max() < 5e-4 * float(oracle["r4"].std())


def test_a_request_that_starts_again_starts_from_empty_states(tmp_path_factory, cpu_kernels):
    d, cfg, w, reqs, oracle = model_and_oracle("S", tmp_path_factory)
    steps = traces.preempted(reqs)
    ps = PAGE_SIZES["S"]
    runner = ModelRunner(load_model(d, torch.float32, "cpu"), ps, traces.peak_tokens(steps) // ps, 3, device="cpu")
    seen = 0
    for rid, pos, row in traces.run_trace_by_position(runner, steps):
        assert (row.double() - oracle[rid][pos]).abs().max() < 5e-4 * float(oracle[rid].std()), (rid, pos)
        seen += 1
    assert seen > sum(len(t) for t in reqs.values())          # the victim's first half came out twice


def test_no_request_grows_beyond_the_position_table(tmp_path, cpu_kernels):
    d = make_model_dir("L", root=str(tmp_path))
    runner = ModelRunner(load_model(d, torch.float32, "cpu"), 4, 200, 1, device="cpu")
    runner.step([StepEntry("a", [1] * 512, (511,))])
    with pytest.raises(ValueError, match="512"):
        runner.step([StepEntry("a", [1], (0,))])


@pytest.mark.parametrize("pages", [64, 14])
def test_greedy_generation_through_the_engine_and_scheduler(pages, tmp_path_factory, cpu_kernels):
    """The public entry point: prompts of unequal length, portions of eight tokens, and (with 14 pages) so few pages that a
    request is preempted and recomputed (a model whose windows are longer than the requests, so that no page goes back early)."""
    d = make_model_dir("F", seed=3, root=str(tmp_path_factory.mktemp("gen")), sigma=0.3)
    cfg, w = read_model(d)
    prompts = [[5, 17, 3, 150, 9, 1, 1, 44, 102, 7, 7], [42] * 19, [7]]
    ref = [plain.generate_greedy(cfg, w, p, 10) for p in prompts]
    assert all(len(set(r)) >= 3 for r in ref), "the continuation is too uniform to test anything"
    eng = Engine(d, dtype="float32", device="cpu", page_size=4, num_pages=pages, num_slots=3, chunked_prefill_size=8,
                 max_num_batched_tokens=16, cuda_graph=False)
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=10, ignore_eos=True))
    assert [o.token_ids for o in outs] == ref
    if pages == 14:
        assert sum(o.preemptions for o in outs) > 0
    eng.runner.cache.check()


@pytest.mark.parametrize("name", ["S", "R"])
def test_generation_with_states_of_looped_layers_and_without_a_paged_cache(name, tmp_path_factory, cpu_kernels):
    d = make_model_dir(name, seed=3, root=str(tmp_path_factory.mktemp("gen")), sigma=0.3)
    cfg, w = read_model(d)
    prompts = [[5, 6, 7, 8], [9] * 12, [3], [100, 2, 50]]
    eng = Engine(d, dtype="float32", device="cpu", page_size=4, num_pages=16, num_slots=2, chunked_prefill_size=8,
                 max_num_batched_tokens=16, cuda_graph=False)
    assert len(eng.runner.cache.states) == 2
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=6, ignore_eos=True))
    assert [o.token_ids for o in outs] == [plain.generate_greedy(cfg, w, p, 6) for p in prompts]
