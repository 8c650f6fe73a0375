"""Dabilorn without a GPU: the configuration reader and what it refuses, the model as the registry builds it (caches that keep a
chunk, a state row that holds the input convolution's memory in front of the mixer's), the plain implementation's own checks (each
mechanism against its sum written out or on made-up inputs), the stretched frequencies, and the engine around the kernels (cache
pages, state slots, step function, scheduler) under every way of cutting the work, with the kernels replaced by their torch
statements."""
import copy
import math

import pytest
import torch

import plain_dabilorn as plain
import traces
from arle_b200 import Engine
from arle_b200.cache import CacheManager
from arle_b200.config import ConfigError, DabilornConfig, config_from_dict, load_config
from arle_b200.engine import ModelRunner, StepEntry, load_model
from arle_b200.parts import AttentionSpec, CacheNeed, Rotary, RotarySpec, RotaryStretch, RoutedExpertsSpec, build_model, build_part
from arle_b200.sampling import SamplingParams
from tiny_dabilorn import CONFIGS, PAGE_SIZES, make_model_dir, read_model

LENGTHS = {"D1": [1, 5, 12, 23, 70, 33], "D2": [2, 17, 40, 64, 9, 31], "A": [1, 20, 33, 7], "W": [3, 30, 11, 2, 45]}
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
    cfg = config_from_dict(CONFIGS["D1"])
    assert isinstance(cfg, DabilornConfig) and [l.type for l in cfg.layers] == ["latent_attention", "attention", "wkv", "attention"]
    lat, a, w, b = cfg.layers
    assert [lat.m(k) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "rot_dims", "rot_base")] == [3, 8, 4, 12, 20, 28, 4, 500.0]
    assert lat.m("stretch") == (4.0, 64.0, 8.0, 1.0) and lat.m("scale") == 0.3
    assert [a.m(k) for k in ("heads", "kv_heads", "dim", "vdim", "chunk", "rot_dims")] == [4, 2, 12, 20, 7, 8] and a.m("stretch") is None
    assert [w.m(k) for k in ("heads", "dim", "decay_rank")] == [3, 8, 5] and b.mlp is None
    assert (lat.mlp.experts, lat.mlp.top, lat.mlp.ff, lat.mlp.shared_ff) == (6, 2, 40, 24) and a.mlp.shared_ff == 0
    assert cfg.norm_eps == 1e-5 and cfg.taps == 4
    d2 = config_from_dict(CONFIGS["D2"])
    assert d2.layers[3].m("chunk") is None and d2.layers[3].m("rot_dims") == 0 and d2.layers[6].m("stretch") is None and d2.layers[6].m("dim") == 0


def test_the_decays_inner_size_comes_from_its_tensor(tmp_path):
    import json
    import os
    d = make_model_dir("W", root=str(tmp_path))
    path = os.path.join(d, "config.json")
    with open(path) as f:
        cfg = json.load(f)
    for l in cfg["layers"]:
        l["mixer"].pop("decay_rank", None)
    with pytest.raises(ConfigError, match="decay"):
        config_from_dict(cfg)
    with open(path, "w") as f:
        json.dump(cfg, f)
    assert [l.m("decay_rank") for l in load_config(d).layers] == [8, 12]


def test_model_spec_norms_caches_and_packed_states():
    spec = config_from_dict(CONFIGS["D1"]).to_model_spec()
    assert spec.head_name is None and spec.embed_norm is not None
    model = build_model(spec)
    needs = model.cache_needs
    assert needs[0].arrays() == ((1, 24),) and needs[0].chunk is None and needs[0].window is None
    assert needs[1].arrays() == ((2, 12), (2, 20)) and needs[1].chunk == 7
    assert needs[2].arrays() == ((1, 8), (1, 8)) and needs[2].chunk == 10
    # every layer remembers three residual rows of 64; the third also its memories (3 x 8 x 8) and the previous token's row
    assert [n.shape for n in model.state_needs] == [(192,), (192,), (192 + 192 + 64,), (192,)]
    names = {d.name for d in model.weight_decls()}
    assert {"embed", "embed.norm", "final.norm", "l0.norm1", "l0.norm2", "l0.ls1", "l0.ls2", "l0.canon1", "l0.mix.dq", "l0.mix.dq.norm", "l0.mix.uq",
            "l0.mix.dkv", "l0.mix.dkv.norm", "l0.mix.uk", "l0.mix.uv", "l0.mix.g", "l0.mix.o", "l1.mix.q.norm", "l1.mix.k.norm", "l1.mix.pb", "l1.mix.g",
            "l2.mix.mu.r", "l2.mix.mu.w", "l2.mix.w1", "l2.mix.w2", "l2.mix.w0", "l2.mix.u", "l2.mix.norm", "l0.mlp.router", "l0.mlp.e5.up",
            "l0.mlp.e5.down", "l0.mlp.shared.up", "l0.mlp.shared.down", "l0.mlp.shared.sg", "l3.ls1", "l3.canon1"} <= names
    assert not any(n.startswith(("head", "l3.norm2", "l3.ls2", "l3.mlp", "l1.mlp.shared", "l2.mix.pb")) or n.endswith(".gate") for n in names)
    d2 = build_model(config_from_dict(CONFIGS["D2"]).to_model_spec())
    assert [n.shape for n in d2.state_needs] == [(20 * 20 + 48,), (5 * 16 + 48,)]           # one tap: the convolutions keep nothing


@pytest.mark.parametrize("change,match", [
    (lambda c: c["layers"][0].update(type="mamba2"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mixer"].update(kv_rank=600), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0), "scaling"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][0]["mixer"].update(dim=0, rot_dim=0, rot=None), "dim"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(scaling={"factor": 2.0}), "scaling"),
    (lambda c: c["layers"][1]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3), "heads"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][2]["mixer"].pop("decay_rank"), "decay"),
    (lambda c: c["layers"][2]["mixer"].update(dim=0), "dim"),
    (lambda c: c["layers"][0].update(mlp={"kind": "dense", "ff": 8}), "mlp"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "chosen"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["canon"].update(taps=0), "canon.taps"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"),
])
def test_configuration_errors_name_the_key(change, match):
    c = copy.deepcopy(CONFIGS["D1"])
    change(c)
    with pytest.raises(ConfigError, match=match):
        config_from_dict(c)


def test_parts_refuse_what_their_kernels_do_not_do():
    base = dict(prefix="p.", hidden_size=32, num_heads=2, num_kv_heads=1, head_dim=8, scale=1.0, qk_norm_eps=1e-5, position=None)
    for bad in (dict(weights="sigmoid"), dict(chunk=4), dict(out_gate=True), dict(qk_norm="row", chunk=4, window=3), dict(qk_norm="row", weights="relu"),
                dict(qk_norm="row", head_gate=True, out_gate=True), dict(qk_norm="row", position=RotarySpec(8, 100.0, stretch=RotaryStretch(4.0, 64, 8, 1)))):
        with pytest.raises(ValueError):
            build_part(AttentionSpec(**dict(base, **bad)))
    for bad in (dict(gated=False, activation="silu"), dict(activation="square_relu"), dict(weight_on="both")):
        with pytest.raises(ValueError):
            build_part(RoutedExpertsSpec(prefix="m.", hidden_size=32, num_experts=4, top=2, expert_ff=8, **bad))


@pytest.mark.parametrize("base,dims,factor,original,fast,slow", [(10000.0, 64, 4.0, 4096, 32.0, 1.0), (500.0, 4, 4.0, 64, 8.0, 1.0), (1e6, 12, 2.0, 900, 16.0, 2.0),
                                                                 (90.0, 6, 0.5, 3000, 1e6, 1e5), (10000.0, 8, 1.0, 512, 4.0, 2.0), (30.0, 16, 8.0, 100000, 2.0, 0.001),
                                                                 (5e5, 128, 40.0, 4096, 1.0, 1.0)])
def test_stretched_frequencies_equal_the_plain_statement(base, dims, factor, original, fast, slow):
    rot = Rotary(RotarySpec(rotary_dim=dims, theta=base, stretch=RotaryStretch(factor, original, fast, slow)))
    rot.load({}, torch.float32, torch.device("cpu"))
    f, amp = plain.stretched_frequencies(base, dims, factor, original, fast, slow)
    torch.testing.assert_close(rot.inv_freq.double(), f, rtol=1e-6, atol=0)
    assert abs(rot.amplitude - amp) < 1e-12
    plain_f = plain.frequencies(base, dims)
    assert (f <= plain_f * max(1.0, 1.0 / factor) + 1e-15).all() and (f >= plain_f * min(1.0, 1.0 / factor) - 1e-15).all()


# ------------------------------------------------------------ the plain implementation
def _rand(g, *shape):
    return torch.randn(*shape, generator=g, dtype=F64)


def test_plain_wkv_memory_equals_its_sum_written_out():
    """o_t = (r_t . (u * k_t)) v_t + sum_(s < t) (r_t . (w_(s+1) * .. * w_(t-1) * k_s)) v_s per head."""
    g = torch.Generator().manual_seed(0)
    T, H, D, Dv = 8, 2, 5, 4
    r, k, v, u = _rand(g, T, H, D), _rand(g, T, H, D), _rand(g, T, H, Dv), _rand(g, H, D)
    w = torch.rand(T, H, D, generator=g, dtype=F64)
    got = plain.wkv_memory(r, k, v, w, u)
    for h in range(H):
        for t in range(T):
            want = (r[t, h] @ (u[h] * k[t, h])) * v[t, h]
            for s in range(t):
                want = want + (r[t, h] @ (w[s + 1: t, h].prod(0) * k[s, h])) * v[s, h]
            assert torch.allclose(got[t, h], want, atol=1e-12)


def test_plain_convolution_mask_rotation_and_norm_on_made_up_inputs():
    g = torch.Generator().manual_seed(1)
    h, w = _rand(g, 6, 3), _rand(g, 3, 4)
    y = plain.plus_short_conv(h, w)
    assert torch.allclose(y[0], h[0] + w[:, 3] * h[0])
    assert torch.allclose(y[4], h[4] + w[:, 0] * h[1] + w[:, 1] * h[2] + w[:, 2] * h[3] + w[:, 3] * h[4])
    see = plain.causal(12, 5)
    assert see[9].nonzero().flatten().tolist() == [5, 6, 7, 8, 9] and see[10].nonzero().flatten().tolist() == [10] and see[4].sum() == 5
    assert plain.causal(5)[4].all() and not plain.causal(5)[2, 3]
    x, pos = _rand(g, 5, 2, 8), torch.arange(5)
    f = plain.frequencies(100.0, 4)
    a = 3 * 100.0 ** (-2 * 1 / 4)
    halves, pairs = plain.rotate(x, pos, f, False), plain.rotate(x, pos, f, True, 1.5)
    assert torch.equal(halves[..., 4:], x[..., 4:]) and torch.allclose(halves[0], x[0])
    assert torch.allclose(halves[3, 1, 1], x[3, 1, 1] * math.cos(a) - x[3, 1, 3] * math.sin(a))
    assert torch.allclose(pairs[3, 0, 3], 1.5 * (x[3, 0, 3] * math.cos(a) + x[3, 0, 2] * math.sin(a))) and torch.allclose(pairs[0, :, :4], 1.5 * x[0, :, :4])
    z = torch.tensor([[1.0, 3.0]], dtype=F64)
    assert torch.allclose(plain.layer_norm(z, torch.tensor([2.0, 5.0]), 0.0), torch.tensor([[-2.0, 5.0]], dtype=F64))
    s = torch.tensor([[0.0, 1.0]], dtype=F64)
    assert torch.allclose(plain.sigmoid_weights(s, torch.tensor([[True, False]]), 0.5), torch.tensor([[1 / (1 + math.exp(-0.5)), 0.0]], dtype=F64))


def test_plain_routing_weights_the_experts_input():
    z = torch.tensor([[0.1, 2.0, -1.0, 2.0, 1.5]], dtype=F64)
    ids, wts = plain.route(z, 3)
    assert ids[0].tolist() == [1, 3, 4] and torch.allclose(wts[0], torch.sigmoid(z[0, ids[0]]))         # ties to the lower index, not renormalised
    g = torch.Generator().manual_seed(2)
    W = {"e.up": _rand(g, 7, 4), "e.down": _rand(g, 4, 7)}
    x = _rand(g, 2, 4)
    # the square of relu: an expert that runs on c x gives c^2 times what it gives for x
    assert torch.allclose(plain.squared_relu_expert(0.3 * x, W, "e."), 0.09 * plain.squared_relu_expert(x, W, "e."))


def test_plain_chunks_and_causality(tmp_path):
    d = make_model_dir("A", seed=5, root=str(tmp_path))
    cfg, w = read_model(d)
    w["l0.canon1"] = torch.zeros_like(w["l0.canon1"])           # so that a position is reached through the attention alone
    toks = traces.make_requests(cfg["vocab"], [40], seed=1)["r0"]
    base = plain.forward(cfg, w, toks)
    # one layer, chunks of 6: position 20 sees 18..20
    for j, reaches in ((2, False), (17, False), (18, True), (19, True), (21, False)):
        moved = list(toks)
        moved[j] = (moved[j] + 1) % cfg["vocab"]
        diff = (plain.forward(cfg, w, moved)[20] - base[20]).abs().max().item()
        assert (diff > 1e-9) == reaches, (j, diff)
    for name in ("D1", "D2"):
        d = make_model_dir(name, seed=5, root=str(tmp_path))
        cfg, w = read_model(d)
        toks = traces.make_requests(cfg["vocab"], [30], seed=1)["r0"]
        assert (plain.forward(cfg, w, toks[:17]) - plain.forward(cfg, w, toks)[:17]).abs().max() < 1e-12


# ------------------------------------------------------------------ the cache manager
def test_the_pages_before_a_requests_chunk_go_back():
    cm = CacheManager([CacheNeed(2, 8, chunk=10), CacheNeed(2, 8, chunk=4), CacheNeed(2, 8, window=10)], [], page_size=4, num_pages=12, max_slots=2,
                      max_tokens_per_request=200, dtype=torch.float32, device="cpu")
    assert len(cm.groups) == 3
    cm.add_request("a")
    seen = []
    for _ in range(30):
        cm.append([("a", 1)])
        cm.release_passed("a")
        cm.check()
        seen.append([g.pool.num_pages - g.pool.num_free for g in cm.groups])
    # 9 tokens: the chunk 0..9 is still open (3 pages); 10 tokens: the next token starts a chunk at 10, pages 0 and 1 are done and
    # page 2 (8..11) stays; 19 tokens: 8..19; 20 tokens: the next chunk starts at a page's start, nothing is held
    assert [s[0] for s in (seen[8], seen[9], seen[18], seen[19], seen[20], seen[29])] == [3, 1, 3, 0, 1, 1]
    assert [s[1] for s in (seen[2], seen[3], seen[4], seen[7])] == [1, 0, 1, 0]
    cm.free_request("a")
    cm.check()
    assert all(g.pool.num_free == g.pool.num_pages for g in cm.groups)


# ------------------------------------------------------------------ the engine on the CPU
@pytest.mark.parametrize("cut", ["whole", "tail_decode", "portions", "mixed"])
@pytest.mark.parametrize("name", ["D1", "D2", "A"])
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


def test_a_request_that_starts_again_starts_from_empty_states(tmp_path_factory, cpu_kernels):
    d, cfg, w, reqs, oracle = model_and_oracle("W", tmp_path_factory)
    steps = traces.preempted(reqs)
    runner = ModelRunner(load_model(d, torch.float32, "cpu"), PAGE_SIZES["W"], 40, 3, device="cpu")
    assert not runner.cache.groups
    seen = 0
    for rid, pos, row in traces.run_trace_by_position(runner, steps):
        assert (row.double() - oracle[rid][pos]).abs().max() < 5e-4 * float(oracle[rid].std()), (rid, pos)
        seen += 1
    assert seen > sum(len(t) for t in reqs.values())          # the victim's first half came out twice


@pytest.mark.parametrize("pages", [64, 14])
def test_greedy_generation_through_the_engine_and_scheduler(pages, tmp_path_factory, cpu_kernels):
    """The public entry point: prompts of unequal length, portions of eight tokens, and (with 14 pages) so few pages that a
    request is preempted and recomputed, cache, states and all."""
    d = make_model_dir("F", seed=3, root=str(tmp_path_factory.mktemp("gen")), branches=4.0)
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


def test_a_wanted_token_in_a_portion_and_the_held_pages(tmp_path_factory, cpu_kernels):
    d, cfg, w, reqs, oracle = model_and_oracle("D1", tmp_path_factory)
    runner = ModelRunner(load_model(d, torch.float32, "cpu"), 4, 40, 2, device="cpu")
    toks = reqs["r4"]
    runner.step([StepEntry("a", toks[:50], ())])
    # the latents keep all 13 pages; chunks of 7: the next token is in 49..55 (page 12 on); chunks of 10: in 50..59 (page 12 on)
    assert [g.pool.num_pages - g.pool.num_free for g in runner.cache.groups] == [13, 1, 1]
    lg = runner.step([StepEntry("a", toks[50:], (0, 5, 19))])
    assert (lg.double() - oracle["r4"][[50, 55, 69]]).abs().max() < 5e-4 * float(oracle["r4"].std())
