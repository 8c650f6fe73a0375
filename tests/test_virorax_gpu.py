"""Virorax on the GPU against the plain implementation (``plain_virorax``): every new or widened kernel alone at sizes of no
model (the position table and the kept embedding output, the factor and the extra rows of the residual sum in the norm and in
the weight-streaming product, biases and partial rotations in the preparation kernels, a sink score per head and a gate per head
in the five attention kernels, the decode launch that prepares, stores, attends and gates, memories with rotated keys continuing
from states in permuted slots token by token and in chunks), the engine under every cutting in float32 and bfloat16 on tiny
configurations, the first tokens of a sequence and prompts that end on page borders, keys just inside and just outside a window
and the sinks made to decide the logits (sharpened attention), a far token living on in the memories, loops, long decoding while
window pages turn over, a request that starts again, greedy generation through the public entry point with CUDA graphs and
preemption, and the replay tool and the command line as subprocesses."""
import copy
import json
import math
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import kernel_refs
import plain_virorax as plain
import traces
from arle_b200 import Engine, ops
from arle_b200.engine import ModelRunner, StepEntry, load_model
from arle_b200.engine.batch import Workspace
from arle_b200.sampling import SamplingParams
from arle_b200.weights import SafetensorsFile, write_safetensors
from tiny_virorax import CONFIGS, PAGE_SIZES, make_model_dir, read_model

pytestmark = pytest.mark.gpu
DEV = "cuda"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16]
IDS = ["f32", "bf16"]
# error of a logits row as a fraction of the spread of the plain model's logits: float32 rounding through a few layers.
# In bfloat16 the engine's worst position may be off by 4.5 times what the plain model's worst is off by when every
# activation it stores is rounded to bfloat16: two ways of rounding the same sums differ by more than either differs
# from the exact result.
REL = {torch.float32: 5e-4, torch.bfloat16: 1e-2}
LENGTHS = {"V1": [1, 5, 12, 23, 70, 130, 33], "V2": [2, 17, 40, 96, 64, 31], "V3": [3, 66, 150, 64, 40, 97], "R": [2, 33, 80, 17, 64],
           "A": [3, 50, 64, 29], "L": [1, 40, 33, 7, 70], "S": [2, 33, 80, 17, 64]}
_cache, _rounding = {}, {}


def rounding_cost(cfg, w, toks, exact) -> float:
    return (plain.forward(cfg, w, toks, rnd=plain.round_bf16) - exact).abs().max().item()


def model_and_oracle(name, tmp_path_factory):
    if name not in _cache:
        d = make_model_dir(name, seed=21, root=str(tmp_path_factory.mktemp(f"tiny{name}")))
        cfg, w = read_model(d)
        reqs = traces.make_requests(cfg["vocab"], LENGTHS[name], seed=6)
        oracle = {r: plain.forward(cfg, w, t) for r, t in reqs.items()}
        _cache[name] = (d, cfg, w, reqs, oracle)
        _rounding[id(oracle)] = max(rounding_cost(cfg, w, t, oracle[r]) for r, t in reqs.items())
    return _cache[name]


def assert_close(got, want, dtype, what="", rounding=0.0):
    err = (got.double().cpu() - want).abs().max(dim=-1).values
    tol = REL[dtype] * float(want.std())
    if dtype == torch.bfloat16:
        tol = max(tol, 4.5 * rounding)
    assert err.max().item() <= tol, f"{what}: first wrong position {int((err > tol).nonzero()[0])}, error {err.max().item():.3g}, tolerance {tol:.3g}"


def _tol(dtype):
    return dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)


def _both(fn, args, outs, kwargs=None):
    """Runs ``fn`` of ops on the GPU and of kernel_refs on the CPU on copies of the same arguments; returns the named outputs
    (positions among ``args``, or names among ``kwargs``)."""
    def on(a, dev):
        if isinstance(a, torch.Tensor):
            return a.to(dev) if dev else a.clone()
        if isinstance(a, tuple):
            return tuple(on(x, dev) for x in a)
        return a
    kwargs = kwargs or {}
    cpu, gpu = [on(a, None) for a in args], [on(a, DEV) for a in args]
    kcpu, kgpu = {k: on(a, None) for k, a in kwargs.items()}, {k: on(a, DEV) for k, a in kwargs.items()}
    getattr(ops, fn)(*gpu, **kgpu)
    getattr(kernel_refs, fn)(*cpu, **kcpu)
    torch.cuda.synchronize()
    return [((kgpu[i] if isinstance(i, str) else gpu[i]).float().cpu(), (kcpu[i] if isinstance(i, str) else cpu[i]).float()) for i in outs]


def _rows(g, starts, lens, ps, extra_pages=5):
    """Rows in scattered pages: positions, row of token, block table, slots of the step's tokens, q_indptr."""
    need = [-(-(s + n) // ps) for s, n in zip(starts, lens)]
    pages = sum(need) + extra_pages
    perm = torch.randperm(pages, generator=g)[: sum(need)].to(torch.int32)
    bt = torch.full((len(lens), max(need)), -1, dtype=torch.int32)
    at = 0
    for r, n in enumerate(need):
        bt[r, :n] = perm[at: at + n]
        at += n
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, lens)]).to(torch.int32)
    row = torch.cat([torch.full((n,), r) for r, n in enumerate(lens)]).to(torch.int32)
    slots = (bt[row.long(), (pos // ps).long()] * ps + pos % ps).to(torch.int32)
    indptr = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32)
    return pages, bt, pos, row, slots, indptr


def _freq(base, dims):
    return torch.pow(torch.tensor(float(base)), -torch.arange(dims // 2) * 2.0 / max(dims, 1)).float()


# ------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("T,H,V", [(5, 40, 30), (70, 64, 200), (3, 36, 9), (1, 1000, 50)])
def test_embedding_with_positions_and_a_second_copy(dtype, T, H, V):
    g = torch.Generator().manual_seed(H)
    ids = torch.randint(0, V, (T,), generator=g).to(torch.int32)
    pos = torch.randint(0, 77, (T,), generator=g).to(torch.int32)
    table, ptab = torch.randn(V, H, generator=g).to(dtype), torch.randn(77, H, generator=g).to(dtype)
    for kw in (dict(pos_table=ptab, positions=pos, out2=torch.zeros(T, H), scale=1.5), dict(pos_table=ptab, positions=pos), dict(out2=torch.zeros(T, H))):
        for got, want in _both("embedding", [ids, table, torch.zeros(T, H)], [2] + (["out2"] if "out2" in kw else []), kw):
            torch.testing.assert_close(got, want, rtol=1e-6, atol=1e-6)
    # a position outside the table writes zeros and raises the flag
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    bad, out = pos.clone(), torch.ones(T, H, device=DEV)
    bad[0] = 77
    ops.embedding(ids.to(DEV), table.to(DEV), out, err, pos_table=ptab.to(DEV), positions=bad.to(DEV))
    assert err.item() == 1 and out[0].abs().max().item() == 0 and (T == 1 or out[1:].abs().min(dim=1).values.max().item() >= 0)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("T,H", [(1, 48), (7, 64), (33, 1000), (3, 4096), (5, 130), (2, 30)])
def test_norm_with_a_factor_on_the_branch_and_rows_that_join(dtype, T, H):
    g = torch.Generator().manual_seed(H)
    resid, delta, extra = torch.randn(T, H, generator=g) * 3, torch.randn(T, H, generator=g).to(dtype), torch.randn(T, H, generator=g)
    w = torch.rand(H, generator=g) + 0.5
    for d, kw in ((delta, dict(delta_scale=0.3, extra=extra)), (delta, dict(delta_scale=-1.7)), (None, dict(extra=extra)), (delta, {})):
        for got, want in _both("rmsnorm", [resid, d, None, w, 1e-5, torch.zeros(T, H, dtype=dtype), True], [0, 5], kw):
            torch.testing.assert_close(got, want, **_tol(dtype))
    rows = torch.tensor([T - 1, 0], dtype=torch.int32)
    for got, want in _both("rmsnorm", [resid, delta, rows, w, 1e-5, torch.zeros(2, H, dtype=dtype), False], [0, 5], dict(delta_scale=0.3)):
        torch.testing.assert_close(got, want, **_tol(dtype))
    for d, sc in ((delta, 0.3), (extra, 1.0)):
        (got, want), = _both("residual_add", [resid, d, sc], [0])
        torch.testing.assert_close(got, want, rtol=1e-6, atol=1e-6)


@pytest.mark.parametrize("M,N,K", [(1, 256, 128), (8, 384, 512), (5, 72, 1024), (3, 1024, 16384)])
def test_product_into_the_residual_with_a_factor_and_joining_rows(M, N, K):
    """resid += factor * x W^T + extra, the rounded gain-scaled rows and their squares' sums; then the next product (plain and with the
    square of relu) applies the rows' norm factor."""
    g = torch.Generator().manual_seed(N)
    x = torch.randn(M, K, generator=g).to(torch.bfloat16)
    w = (torch.randn(N, K, generator=g) / math.sqrt(K)).to(torch.bfloat16)
    resid, extra, gain = torch.randn(M, N, generator=g), torch.randn(M, N, generator=g), torch.rand(N, generator=g) + 0.5
    for ex in (extra, None):
        r = resid.to(DEV).clone()
        xs = torch.zeros(M, N, dtype=torch.bfloat16, device=DEV)
        ss = torch.zeros(ops.SS_TABLE_SHAPE, device=DEV)
        sink = ops.ResidualSink(r, gain.to(DEV), 1e-5, xs, ss, 0.37, ex.to(DEV) if ex is not None else None)
        assert ops.gemm(x.to(DEV), w.to(DEV), None, sink=sink) is True
        want = resid.double() + 0.37 * (x.double() @ w.double().t()) + (ex.double() if ex is not None else 0.0)
        torch.testing.assert_close(r.cpu().double(), want, rtol=1e-4, atol=1e-4)
        if N % 32 == 0:
            w2 = (torch.randn(96, N, generator=g) / math.sqrt(N)).to(torch.bfloat16)
            out = torch.zeros(M, 96, dtype=torch.bfloat16, device=DEV)
            ops.gemm_square_relu(ops.ScaledRows(xs, ss, 1e-5), w2.to(DEV), out)
            n = want / torch.sqrt((want * want).mean(-1, keepdim=True) + 1e-5) * gain.double()
            torch.testing.assert_close(out.float().cpu(), (torch.relu(n @ w2.double().t()) ** 2).float(), rtol=3e-2, atol=3e-2)
    ops.check_errors(DEV)


@pytest.mark.parametrize("M,N,K", [(1024, 320, 128), (1100, 1000, 256), (4096, 96, 72)])
def test_first_half_of_an_ungated_feed_forward_on_the_two_sm_kernel(M, N, K):
    g = torch.Generator().manual_seed(N)
    x, w = torch.randn(M, K, generator=g).to(torch.bfloat16), (torch.randn(N, K, generator=g) / math.sqrt(K)).to(torch.bfloat16)
    want = torch.relu(x.double() @ w.double().t()) ** 2
    for fn in (lambda out: ops.gemm_tcgen05_pair(x.to(DEV), w.to(DEV), out, activation="square_relu"), lambda out: ops.gemm_square_relu(x.to(DEV), w.to(DEV), out)):
        out = torch.full((M, N), float("nan"), dtype=torch.bfloat16, device=DEV)
        fn(out)
        ops.check_errors(DEV)
        torch.testing.assert_close(out.double().cpu(), want, rtol=1e-2, atol=1e-2)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("nq,nkv,hd,vd,window,ps", [(4, 2, 16, 24, 7, 4), (1, 1, 12, 40, 5, 8), (6, 2, 8, 4, 1, 16), (3, 1, 48, 48, 33, 16),
                                                    (2, 2, 80, 32, 0, 4), (5, 5, 20, 20, 40, 16)])
def test_general_attention_with_a_sink_and_a_gate_per_head(dtype, nq, nkv, hd, vd, window, ps):
    """Sinks far below, among and far above the scores; pages that a window has passed are poisoned."""
    g = torch.Generator().manual_seed(hd + vd + window)
    starts, lens = [0, 2, 60, 119], [70, 9, 1, 12]
    pages, bt, pos, row, slots, _ = _rows(g, starts, lens, ps)
    T = int(pos.numel())
    q = torch.randn(T, nq * hd, generator=g).to(dtype)
    kc, vc = torch.randn(pages, nkv, ps, hd, generator=g).to(dtype), torch.randn(pages, nkv, ps, vd, generator=g).to(dtype)
    if window:
        for r, s in enumerate(starts):
            for p in range(max(0, s - window + 1) // ps):
                kc[bt[r, p]], vc[bt[r, p]] = 1e4, float("nan")
    sinks = torch.linspace(-4.0, 6.0, nq) if nq > 1 else torch.tensor([1.5])
    gate = (torch.randn(T, nq + 5, generator=g) * 2).to(dtype)[:, 3: nq + 3]
    for kw in (dict(sink=sinks, gate=gate), dict(sink=sinks), dict(gate=gate)):
        (got, want), = _both("paged_attention", [q, torch.zeros(T, nq * vd, dtype=dtype), kc, vc, pos, row, bt, nq, nkv, hd, ps, 0.3, window or None], [1],
                             dict(vd=vd, **kw))
        assert torch.isfinite(got).all()
        torch.testing.assert_close(got, want, **_tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("nq,nkv,hd,rdim,ps,norm", [(8, 2, 64, 16, 16, True), (4, 4, 64, 32, 8, True), (4, 1, 128, 128, 16, True), (6, 2, 128, 64, 16, True),
                                                   (2, 1, 128, 8, 16, False), (3, 1, 64, 4, 16, True), (5, 1, 48, 20, 4, True), (12, 4, 64, 64, 16, True),
                                                   (4, 2, 128, 96, 16, True), (2, 2, 64, 0, 16, True), (40, 8, 128, 32, 16, True)])
def test_preparation_with_biases_and_a_partial_rotation(dtype, nq, nkv, hd, rdim, ps, norm):
    """Few tokens (a warp a head) and many (a block a token), with and without the step's table of angles."""
    g = torch.Generator().manual_seed(hd + rdim)
    for starts, lens in (([0, 13, 200], [9, 4, 1]), ([5, 300], [77, 40])):
        pages, bt, pos, row, slots, _ = _rows(g, starts, lens, ps)
        T = int(pos.numel())
        slots[1] = -1                                      # a token that is not stored
        n = (nq + 2 * nkv) * hd
        wide = torch.randn(T, -(-(n + 8) // 8) * 8, generator=g).to(dtype)
        wq, wk, bias = torch.rand(hd, generator=g) + 0.5, torch.rand(hd, generator=g) + 0.5, torch.randn(n, generator=g)
        inv = _freq(300.0, rdim)
        kc, vc = torch.zeros(pages, nkv, ps, hd, dtype=dtype), torch.zeros(pages, nkv, ps, hd, dtype=dtype)
        angles = torch.zeros(T, rdim // 2, 2)
        if rdim:
            kernel_refs.rotary_angles(pos, inv, angles)
        args = [wide, pos, slots, wq if norm else None, wk if norm else None, 1e-5, inv if rdim else None, rdim, kc, vc, nq, nkv, hd, ps]
        for kw in (dict(bias=bias), dict(bias=bias, angles=angles), dict(), dict(angles=angles)):
            if "angles" in kw and not rdim:
                continue
            for got, want in _both("attention_prep", args, [0, 8, 9], kw):
                torch.testing.assert_close(got, want, **_tol(dtype))
        # the general preparation with values of another width
        vd = hd + 4
        n2 = (nq + nkv) * hd + nkv * vd
        qkv = torch.randn(T, n2, generator=g).to(dtype)
        args = [qkv, pos, slots, wq if norm else None, wk if norm else None, 1e-5 if norm else None, inv if rdim else None, rdim,
                torch.zeros(pages, nkv, ps, hd, dtype=dtype), torch.zeros(pages, nkv, ps, vd, dtype=dtype), nq, nkv, hd, vd, ps]
        for got, want in _both("attention_prep_post", args, [0, 8, 9], dict(norm_first=True, bias=torch.randn(n2, generator=g))):
            torch.testing.assert_close(got, want, **_tol(dtype))


@pytest.mark.parametrize("nq,nkv,hd,ps,window", [(8, 2, 128, 16, 37), (4, 1, 64, 16, 33), (2, 2, 64, 32, 300), (12, 4, 128, 8, 64), (4, 2, 128, 16, None),
                                                 (16, 1, 64, 16, None)])
def test_a_sink_and_a_gate_per_head_in_the_tensor_core_attention_kernels(nq, nkv, hd, ps, window):
    """Prompts on mma.sync and on tcgen05, decoding with split keys and streaming: each against the plain statement, which differs
    from the attention without the sinks, and from the one with every head's sink of its neighbour, by far more than the tolerance."""
    from test_kernels_gpu import _fast_setup

    scale = 2.0 / math.sqrt(hd)
    g = torch.Generator().manual_seed(nq)
    sinks = torch.randn(nq, generator=g) * 2 + 1

    def want(q, kc, vc, pos, rows, bt, sinks_, gate):
        exp = torch.empty(q.shape[0], nq * hd, dtype=torch.bfloat16)
        kernel_refs.paged_attention(q.cpu(), exp, kc.cpu(), vc.cpu(), pos.cpu(), rows.cpu(), bt.cpu(), nq, nkv, hd, ps, scale, window, sink=sinks_,
                                    gate=gate)
        return exp.float()

    lens, q_lens = [130, 300, 128, 129, 9, 700], [130, 2, 128, 3, 1, 333]
    q, kc, vc, pos, rows, bt, qi, kv = _fast_setup(nq, nkv, hd, ps, lens, q_lens, seed=6)
    gate = (torch.randn(q.shape[0], nq + 3, generator=g) * 2).to(torch.bfloat16)
    gcut = gate[:, 2: nq + 2]
    exp = want(q, kc, vc, pos, rows, bt, sinks, gcut)
    for other in (None, sinks.roll(1)):
        assert (exp - want(q, kc, vc, pos, rows, bt, other, gcut)).abs().max() > 0.05
    assert (exp - want(q, kc, vc, pos, rows, bt, sinks, None)).abs().max() > 0.05
    tail = dict(sink=sinks.to(DEV), gate=gate.to(DEV)[:, 2: nq + 2])
    for fn in ([ops.paged_attention_prefill_tc] if hd == 128 and ps % 16 == 0 else []) + [ops.paged_attention_prefill]:
        out = torch.zeros(q.shape[0], nq * hd, dtype=torch.bfloat16, device=DEV)
        fn(q, out, kc, vc, qi, kv, bt, nq, nkv, hd, ps, scale, window, max(q_lens), **tail)
        ops.check_errors(DEV)
        torch.testing.assert_close(out.float().cpu(), exp, rtol=2e-2, atol=1e-2)
    lens = [1, 63, 64, 65, 700, 2049, 17, window or 50]
    R = len(lens)
    q, kc, vc, pos, rows, bt, qi, kv = _fast_setup(nq, nkv, hd, ps, lens, [1] * R, seed=3)
    gate = (torch.randn(R, nq, generator=g) * 2).to(torch.bfloat16)
    exp = want(q, kc, vc, pos, rows, bt, sinks, gate)
    tail = dict(sink=sinks.to(DEV), gate=gate.to(DEV))
    for splits in (1, 2, 5):
        out = torch.zeros(R, nq * hd, dtype=torch.bfloat16, device=DEV)
        po, pml = torch.zeros(R * nq * splits * hd, device=DEV), torch.zeros(R * nq * splits * 2, device=DEV)
        ops.paged_attention_decode(q, out, kc, vc, qi, kv, bt, nq, nkv, hd, ps, scale, window, splits, po, pml,
                                   torch.zeros(R * nkv, dtype=torch.int32, device=DEV), **tail)
        torch.testing.assert_close(out.float().cpu(), exp, rtol=2e-2, atol=1e-2)
    for ctas in (3, 148) if ps % 16 == 0 else ():
        slots = (ctas + R * nkv) * (nq // nkv)
        out = torch.zeros(R, nq * hd, dtype=torch.bfloat16, device=DEV)
        ops.paged_attention_decode_stream(q, out, kc, vc, qi, kv, bt, nq, nkv, hd, ps, scale, window, torch.zeros(slots * hd, device=DEV),
                                          torch.zeros(slots * 2, device=DEV), torch.zeros(R * nkv, dtype=torch.int32, device=DEV), ctas, **tail)
        ops.check_errors(DEV)
        torch.testing.assert_close(out.float().cpu(), exp, rtol=2e-2, atol=1e-2)


@pytest.mark.parametrize("nq,nkv,hd,rdim,ps,window", [(8, 2, 64, 16, 16, 33), (4, 1, 128, 64, 16, 37), (6, 2, 64, 64, 32, None), (16, 1, 128, 128, 16, 100),
                                                      (2, 2, 64, 0, 16, 5), (4, 2, 128, 40, 16, None), (3, 1, 64, 4, 16, 64)])
def test_one_launch_decoding_with_biases_partial_rotation_sinks_and_gates(nq, nkv, hd, rdim, ps, window):
    from test_kernels_gpu import _fast_setup

    g = torch.Generator().manual_seed(hd + rdim)
    lens = [1, 63, 64, 65, 700, 1025, 17, 2, window or 90]
    R, scale = len(lens), 1.5 / math.sqrt(hd)
    _, kc, vc, pos, rows, bt, qi, kv = _fast_setup(nq, nkv, hd, ps, lens, [1] * R, seed=3)
    n = (nq + 2 * nkv) * hd
    qkv = torch.randn(R, -(-(n + nq) // 8) * 8, generator=g).to(torch.bfloat16)
    bias, sinks = torch.randn(n, generator=g), torch.randn(nq, generator=g) + 1
    wq, wk = torch.rand(hd, generator=g) + 0.5, torch.rand(hd, generator=g) + 0.5
    inv = _freq(500.0, rdim)
    slots = torch.tensor([int(bt[r, (l - 1) // ps]) * ps + (l - 1) % ps for r, l in enumerate(lens)], dtype=torch.int32)
    c = [x.cpu().clone() for x in (qkv, kc, vc)]
    kernel_refs.attention_prep(c[0], pos.cpu(), slots, wq, wk, 1e-5, inv if rdim else None, rdim, c[1], c[2], nq, nkv, hd, ps, bias=bias)
    exp = torch.zeros(R, nq * hd, dtype=torch.bfloat16)
    kernel_refs.paged_attention(c[0][:, : nq * hd], exp, c[1], c[2], pos.cpu(), rows.cpu(), bt.cpu(), nq, nkv, hd, ps, scale, window, sink=sinks,
                                gate=qkv[:, n: n + nq])
    for memo in (None, {}):
        batch = SimpleNamespace(max_q_len=1, num_rows=R, ws=Workspace(DEV), q_indptr=qi, kv_lens=kv, memo=memo)
        x, kb, vb = qkv.to(DEV), kc.clone(), vc.clone()
        assert ops.fused_decode_supported(x, batch, kb.dtype, nq, nkv, hd, ps, rdim)
        out = torch.full((R, nq * hd), float("nan"), dtype=torch.bfloat16, device=DEV)
        ops.decode_attention_with_prep(x, out, kb, vb, slots.to(DEV), wq.to(DEV), wk.to(DEV), 1e-5, inv.to(DEV) if rdim else None, bt, nq, nkv, hd, ps,
                                       scale, window, batch, rotary_dim=rdim, bias=bias.to(DEV), sink=sinks.to(DEV), gate=x[:, n: n + nq])
        ops.check_errors(DEV)
        torch.testing.assert_close(kb.float().cpu(), c[1].float(), rtol=1e-2, atol=1e-2)
        torch.testing.assert_close(vb.float().cpu(), c[2].float(), rtol=1e-2, atol=1e-2)
        torch.testing.assert_close(out.float().cpu(), exp.float(), rtol=2e-2, atol=2e-2)


MEMORIES = [(3, 8, 12, 8, [1, 5, 40]), (1, 20, 8, 6, [18, 1, 2]), (4, 64, 64, 32, [33, 1, 9, 200]), (5, 4, 6, 2, [1, 1, 1]), (2, 128, 128, 64, [70, 3, 64, 65]),
            (2, 160, 32, 160, [70, 3]), (4, 32, 100, 0, [300, 128]), (2, 36, 65, 20, [129, 31, 32]), (3, 17, 5, 6, [97, 1])]


@pytest.mark.parametrize("act", ["none", "silu"])
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("H,dim,vdim,rdim,lens", MEMORIES)
def test_rotated_memories_token_by_token_and_in_chunks(dtype, H, dim, vdim, rdim, lens, act):
    """Rows of unequal length that continue from memories in permuted slots at positions far from zero; decays from 0 to 1; the scan
    alone, and the chunks for the long rows with the scan for the others: the same memories and the same outputs."""
    if act == "silu":
        rdim = 0
    g = torch.Generator().manual_seed(dim + vdim)
    T, R = sum(lens), len(lens)
    wide = torch.randn(T, H * (2 * dim + vdim) + 8, generator=g).to(dtype)
    decay = torch.cat([torch.tensor([0.0]), torch.linspace(0.3, 1.0, H - 1)]) if H > 1 else torch.tensor([0.999])
    state = torch.randn(R + 2, H * vdim * dim + 8, generator=g) * 0.5
    slots = torch.randperm(R + 2, generator=g)[:R].to(torch.int32)
    indptr = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32)
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip((0, 40, 700, 3), lens)]).to(torch.int32)
    inv = _freq(1000.0, rdim)
    rot = (pos, inv, rdim) if rdim else None
    cut = (slice(0, H * dim), slice(H * dim, 2 * H * dim), slice(2 * H * dim, H * (2 * dim + vdim)))
    q_scale = dim ** -0.5
    out, st = torch.zeros(T, H, vdim), state.clone()
    kernel_refs.decay_scan(*(wide[:, c] for c in cut), decay, None, st, indptr, slots, out, H, H, dim, vdim, False, q_scale, act=act, rotation=rot)
    x = wide.to(DEV)
    parts = [x[:, c] for c in cut]
    rot = (pos.to(DEV), inv.to(DEV), rdim) if rdim else None
    batch = SimpleNamespace(num_rows=R, q_lens=lens, q_indptr=indptr.to(DEV), state_slots=slots.to(DEV), ws=Workspace(DEV), memo={})
    chunks = ops.decay_chunk_count(lens, dim, dtype)
    assert chunks == (sum(-(-n // 64) for n in lens if n > 32) if dim <= 128 else 0)
    for way in ("scan", "chunks"):
        got, s = torch.zeros(T, H, vdim, device=DEV), state.to(DEV)
        if way == "chunks":
            if not chunks:
                continue
            ops.decay_chunks(*parts, decay.to(DEV), s, batch, got, H, dim, vdim, q_scale, act=act, rotation=rot, chunks=chunks)
        if way == "scan" or min(lens) <= 32:
            ops.decay_scan(*parts, decay.to(DEV), None, s, batch.q_indptr, batch.state_slots, got, H, H, dim, vdim, False, q_scale, act=act, rotation=rot,
                           longest=32 if way == "chunks" else 0)
        # q, k and v are the same numbers for both; float32 sums in another order
        torch.testing.assert_close(got.cpu(), out, rtol=1e-4, atol=2e-4 * float(out.abs().max()))
        torch.testing.assert_close(s.cpu(), st, rtol=1e-4, atol=2e-4)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_unit_heads_with_a_silu_gate(dtype):
    g = torch.Generator().manual_seed(3)
    for T, H, vd in ((5, 3, 12), (3, 1, 128), (70, 4, 32), (2, 5, 7)):
        o = torch.randn(T, H * vd, generator=g) * 3
        gate = torch.randn(T, H * vd + 8, generator=g).to(dtype)[:, 4: H * vd + 4]
        (got, want), = _both("gla_out", [o, gate, None, 1e-5, 1.0, torch.zeros(T, H * vd, dtype=dtype), H, vd], [5], dict(gate_act="silu"))
        torch.testing.assert_close(got, want, **_tol(dtype))


# ------------------------------------------------------------------ the engine under every cutting
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("cut", ["whole", "tail_decode", "portions", "mixed"])
@pytest.mark.parametrize("name", ["V1", "V2", "V3", "R", "S"])
def test_cuttings(name, cut, dtype, tmp_path_factory):
    d, cfg, w, reqs, oracle = model_and_oracle(name, tmp_path_factory)
    steps = traces.mixed(reqs, seed=4) if cut == "mixed" else getattr(traces, cut)(reqs)
    ps = PAGE_SIZES[name]
    runner = ModelRunner(load_model(d, dtype, DEV), ps, max(1, traces.peak_tokens(steps) // ps), 4, device=DEV)
    got = traces.run_trace(runner, steps)
    ops.check_errors(DEV)
    runner.cache.check()
    assert runner.cache.num_free_slots == 4 and all(g.pool.num_free == g.pool.num_pages for g in runner.cache.groups)
    for r, want in oracle.items():
        assert_close(got[r], want, dtype, f"{name} {cut}: request {r}", _rounding[id(oracle)])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_other_page_sizes_and_the_plain_kernel_set(dtype, tmp_path_factory):
    d, cfg, w, reqs, oracle = model_and_oracle("V3", tmp_path_factory)
    steps = traces.mixed(reqs, seed=9)
    for ps, ks in ((32, "fast"), (64, "fast"), (16, "plain")):
        runner = ModelRunner(load_model(d, dtype, DEV), ps, max(1, -(-traces.peak_tokens(steps) // ps)), 4, device=DEV, kernel_set=ks)
        got = traces.run_trace(runner, steps)
        for r, want in oracle.items():
            assert_close(got[r], want, dtype, f"pages of {ps}, {ks} kernels, request {r}", _rounding[id(oracle)])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", ["V1", "V2", "R"])
def test_first_tokens_and_page_borders(name, dtype, tmp_path_factory):
    d, cfg, w, reqs, oracle = model_and_oracle(name, tmp_path_factory)
    ps = PAGE_SIZES[name]
    runner = ModelRunner(load_model(d, dtype, DEV), ps, 64, 3, device=DEV)
    toks = [7, 7, 3, 150, 1]
    want = plain.forward(cfg, w, toks)
    rc = _rounding[id(oracle)]
    one_by_one = torch.cat([runner.step([StepEntry("a", [t], (0,))]).clone() for t in toks])
    together = runner.step([StepEntry("b", toks, range(5))]).clone()
    assert_close(one_by_one, want, dtype, "one by one", rc)
    assert_close(together, want, dtype, "together", rc)
    runner.end_request("a"), runner.end_request("b")
    # prompts that end exactly on a page border, one before and one after, then two decoded tokens
    long = traces.make_requests(cfg["vocab"], [4 * ps + 3], seed=2)["r0"]
    want = plain.forward(cfg, w, long)
    for n in (ps - 1, ps, ps + 1, 2 * ps, 4 * ps):
        got = [runner.step([StepEntry("c", long[:n], range(n))]).clone()]
        got += [runner.step([StepEntry("c", [long[n + i]], (0,))]).clone() for i in range(2)]
        assert_close(torch.cat(got), want[: n + 2], dtype, f"prompt of {n}", rc)
        runner.end_request("c")


def _changed(name, tmp_path, change, length, edit_config=None):
    """A tiny model with some tensors (and configuration values) changed: (folder, config, weights, tokens, the plain logits,
    what rounding costs)."""
    d = make_model_dir(name, seed=9, root=str(tmp_path))
    path = os.path.join(d, "model.safetensors")
    f = SafetensorsFile(path)
    t = {n: f.tensor(n).clone() for n in f.names()}
    change(t)
    write_safetensors(path, t)
    cfg, w = read_model(d)
    if edit_config is not None:
        edit_config(cfg)
        with open(os.path.join(d, "config.json"), "w") as fh:
            json.dump(cfg, fh)
    toks = traces.make_requests(cfg["vocab"], [length], seed=3)["r0"]
    want = plain.forward(cfg, w, toks)
    return d, cfg, w, toks, want, rounding_cost(cfg, w, toks, want)


def _run_cut(d, dtype, ps, toks, sizes):
    runner = ModelRunner(load_model(d, dtype, DEV), ps, -(-(len(toks) + 64) // ps), 2, device=DEV)
    got, at = [], 0
    for n in sizes:
        got.append(runner.step([StepEntry("r", toks[at:at + n], range(n))]).clone())
        at += n
    assert at == len(toks)
    return torch.cat(got)


def _scale(t, name, f):
    t[name] = (t[name].float() * f).to(torch.bfloat16)


CUTS_90 = ((90,), (40, 1, 1, 5, 2, 13, 6, 7) + (1,) * 15, (2,) * 10 + (3, 4, 12, 13, 14) + (1,) * 24)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_keys_at_the_windows_edges_and_the_sinks_decide_the_logits(dtype, tmp_path):
    """Random weights make attention nearly uniform, which hides a window that is one token off.  The score scale is raised until
    the softmax picks single keys, and the sinks are set among the scores, another for each head.  The plain model with the window
    one longer or one shorter, without the sinks, with the heads' sinks swapped, without the gate's or the projections' biases is
    far from the plain model at several positions; the engine is not, in prompts cut at every kind of place and in decoding."""
    def change(t):
        t["l0.mix.sink"] = torch.tensor([3.0, -1.0], dtype=torch.bfloat16)
        for n in "qkv":
            _scale(t, f"l0.mix.{n}.b", 4.0)
        _scale(t, "l0.mix.g", 4.0)

    d, cfg, w, toks, want, rc = _changed("A", tmp_path, change, 90, lambda cfg: cfg["layers"][0]["mixer"].update(scale=2.5))
    tol = max(REL[dtype] * float(want.std()), 4.5 * rc if dtype == torch.bfloat16 else 0.0)

    def shows(what, cfg_, w_):
        wrong = (plain.forward(cfg_, w_, toks) - want).abs().max(dim=-1).values
        assert (wrong > 3 * tol).sum() >= 2, f"{what} would not show"

    for delta in (1, -1):
        off = copy.deepcopy(cfg)
        off["layers"][0]["mixer"]["mask"]["size"] += delta
        shows(f"a window off by {delta}", off, w)
    shows("a softmax without sinks", cfg, dict(w, **{"l0.mix.sink": torch.full((2,), -100.0, dtype=torch.float64)}))
    shows("sinks of the wrong heads", cfg, dict(w, **{"l0.mix.sink": w["l0.mix.sink"].flip(0)}))
    shows("a gate of one half", cfg, dict(w, **{"l0.mix.g": 0 * w["l0.mix.g"]}))
    for n in "qkv":
        shows(f"no bias on {n}", cfg, dict(w, **{f"l0.mix.{n}.b": 0 * w[f"l0.mix.{n}.b"]}))
    for sizes in CUTS_90:
        assert_close(_run_cut(d, dtype, PAGE_SIZES["A"], toks, sizes), want, dtype, f"cut {sizes[:4]}", rc)


@pytest.mark.parametrize("hd,rot", [(64, 32), (128, 128), (128, 32)])
def test_sharp_windows_and_sinks_on_the_tensor_core_kernels(hd, rot, tmp_path):
    """The same with heads of 64 and 128 in bfloat16, where prompts run on the tensor-core kernels and decoded tokens in the launch
    that prepares, stores, attends and gates."""
    cfg0 = copy.deepcopy(CONFIGS["A"])
    cfg0["layers"][0]["mixer"].update(heads=4, kv_heads=2, dim=hd, vdim=hd, scale=4.8 / math.sqrt(hd), mask={"size": 21}, rot={"base": 3000.0, "dims": rot})
    from arle_b200.weights import write_random_model

    d = write_random_model(str(tmp_path / "m"), cfg0, 5, sigma=0.12, gain_jitter=0.3)
    path = os.path.join(d, "model.safetensors")
    f = SafetensorsFile(path)
    t = {n: f.tensor(n).clone() for n in f.names()}
    t["l0.mix.sink"] = torch.tensor([8.0, -1.0, 12.0, 5.0], dtype=torch.bfloat16)
    write_safetensors(path, t)
    cfg, w = read_model(d)
    toks = traces.make_requests(cfg["vocab"], [90], seed=3)["r0"]
    want = plain.forward(cfg, w, toks)
    rc = rounding_cost(cfg, w, toks, want)
    tol = max(REL[torch.bfloat16] * float(want.std()), 4.5 * rc)
    for delta in (1, -1):
        off = copy.deepcopy(cfg)
        off["layers"][0]["mixer"]["mask"]["size"] += delta
        assert ((plain.forward(off, w, toks) - want).abs().max(dim=-1).values > 2 * tol).sum() >= 1, f"window off by {delta} would not show"
    nosink = dict(w, **{"l0.mix.sink": torch.full((4,), -100.0, dtype=torch.float64)})
    assert ((plain.forward(cfg, nosink, toks) - want).abs().max(dim=-1).values > 3 * tol).sum() >= 2
    for sizes in CUTS_90:
        assert_close(_run_cut(d, torch.bfloat16, 16, toks, sizes), want, torch.bfloat16, f"cut {sizes[:4]}", rc)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_a_far_token_lives_on_in_the_memories(dtype, tmp_path):
    """Decays of 0.999 and 1: the memories keep what the first tokens wrote for hundreds of steps.  A memory that is lost, reset
    or mixed up between steps shows; so do keys that are not rotated and a decay that is a little off."""
    d, cfg, w, toks, want, rc = _changed("R", tmp_path, lambda t: None, 330)
    tol = max(REL[dtype] * float(want.std()), 4.5 * rc if dtype == torch.bfloat16 else 0.0)
    moved = list(toks)
    moved[5] = (moved[5] + 1) % cfg["vocab"]
    assert (plain.forward(cfg, w, moved)[200:] - want[200:]).abs().max().item() / float(want.std()) > 1e-2, "the memories do not remember far tokens"
    for key, value in (("rot", None), ("decay", [0.98, 1.0])):
        off = copy.deepcopy(cfg)
        off["layers"][0]["mixer"][key] = value
        assert ((plain.forward(off, w, toks) - want).abs().max(dim=-1).values > 2 * tol).sum() >= 2, key
    for sizes in ((330,), (130, 1, 1, 64, 2, 99, 1, 1) + (1,) * 31, (33, 2, 65, 64, 3, 128, 35)):
        assert_close(_run_cut(d, dtype, PAGE_SIZES["R"], toks, sizes), want, dtype, f"cut {sizes[:4]}", rc)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_passes_of_a_loop_keep_caches_and_states_of_their_own(dtype, tmp_path_factory):
    """One layer run four times: another number of passes, or passes without the embedding output added before them, are far off."""
    d, cfg, w, reqs, oracle = model_and_oracle("L", tmp_path_factory)
    rc = _rounding[id(oracle)]
    for off in (dict(cfg, loop={"start": 0, "stop": 1, "times": 3}), {k: v for k, v in dict(cfg, layers=cfg["layers"] * 4).items() if k != "loop"}):
        ww = dict(w, **{f"l{i}." + n[3:]: w[n] for i in range(1, 4) for n in w if n.startswith("l0.")})
        wrong = (plain.forward(off, ww, reqs["r4"]) - oracle["r4"]).abs().max().item()
        assert wrong > 3 * max(4.5 * rc, REL[dtype] * float(oracle["r4"].std()))
    for steps in (traces.tail_decode(reqs, 20), traces.mixed(reqs, seed=2)):
        runner = ModelRunner(load_model(d, dtype, DEV), 4, traces.peak_tokens(steps) // 4, 4, device=DEV)
        assert len(runner.model.cache_needs) == 4
        got = traces.run_trace(runner, steps)
        for r, want in oracle.items():
            assert_close(got[r], want, dtype, f"request {r}", rc)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_long_decoding_keeps_cache_and_states_exact(dtype, tmp_path_factory):
    d, cfg, w, reqs, oracle = model_and_oracle("V1", tmp_path_factory)
    toks = traces.make_requests(cfg["vocab"], [320], seed=8)["r0"]
    want = plain.forward(cfg, w, toks)
    runner = ModelRunner(load_model(d, dtype, DEV), 4, 80, 2, device=DEV)         # pages of four: the windows' pages turn over
    got = [runner.step([StepEntry("r", toks[:20], range(20))]).clone()]
    got += [runner.step([StepEntry("r", [t], (0,))]).clone() for t in toks[20:]]
    assert [g.pool.num_pages - g.pool.num_free for g in runner.cache.groups] == [2, 3]
    assert_close(torch.cat(got), want, dtype, "300 decoded tokens", rounding_cost(cfg, w, toks, want))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_a_request_that_starts_again(dtype, tmp_path_factory):
    d, cfg, w, reqs, oracle = model_and_oracle("S", tmp_path_factory)
    steps = traces.preempted(reqs)
    ps = PAGE_SIZES["S"]
    runner = ModelRunner(load_model(d, dtype, DEV), ps, traces.peak_tokens(steps) // ps, 3, device=DEV)
    for rid, pos, row in traces.run_trace_by_position(runner, steps):
        assert_close(row[None], oracle[rid][pos][None], dtype, f"{rid} at {pos}", _rounding[id(oracle)])


@pytest.mark.parametrize("name", ["V3", "S"])
def test_a_batch_of_decoded_tokens_wider_than_the_weight_streaming_product(name, tmp_path_factory):
    """Eleven requests decoded together, captured and kernel by kernel, against each alone (eight rows and fewer run on fused products)."""
    d, cfg, w, _, _ = model_and_oracle(name, tmp_path_factory)
    reqs = traces.make_requests(cfg["vocab"], [5 + 7 * i for i in range(11)], seed=4)
    oracle = {r: plain.forward(cfg, w, t) for r, t in reqs.items()}
    rc = max(rounding_cost(cfg, w, t, oracle[r]) for r, t in reqs.items())
    for dtype in DTYPES:
        for graphs in (False, True):
            runner = ModelRunner(load_model(d, dtype, DEV), 16, 80, 11, device=DEV)
            if graphs:
                runner.enable_graphs()
            runner.step([StepEntry(r, t[:-3], ()) for r, t in reqs.items()])
            for back in (3, 2, 1):
                lg = runner.step([StepEntry(r, [t[-back]], (0,)) for r, t in reqs.items()])
                for i, (r, t) in enumerate(reqs.items()):
                    assert_close(lg[i][None].clone(), oracle[r][len(t) - back][None], dtype, f"{r}, {back} before the end", rc)
            assert (runner.graph_steps > 0) == graphs


# ------------------------------------------------------------------ generation
@pytest.mark.parametrize("graph", [True, False], ids=["graphs", "eager"])
@pytest.mark.parametrize("name", ["F", "V1", "R", "S"])
def test_greedy_generation_equals_plain_model_f32(name, graph, tmp_path):
    d = make_model_dir(name, seed=3, root=str(tmp_path), sigma=0.3)
    cfg, w = read_model(d)
    prompts = [[5, 17, 3, 150, 9, 1, 1, 44, 102, 7, 7], [42] * 19, [7], list(range(20, 61))]
    ref = [plain.generate_greedy(cfg, w, p, 12) for p in prompts]
    assert all(len(set(r)) >= 3 for r in ref), "the continuation is too uniform to test anything"
    ps = PAGE_SIZES[name]
    for pages in (256 // ps, 112 // ps):                     # plenty; and (for the long window) so few that a request is preempted
        eng = Engine(d, dtype="float32", device=DEV, page_size=ps, num_pages=pages, num_slots=3, chunked_prefill_size=16,
                     max_num_batched_tokens=32, cuda_graph=graph)
        outs = eng.generate(prompts, SamplingParams(max_new_tokens=12, ignore_eos=True))
        assert [o.token_ids for o in outs] == ref, f"{pages} pages"
        assert not graph or eng.runner.graph_steps > 0
        eng.runner.cache.check()


def test_greedy_generation_bf16_stays_on_the_plain_models_best(tmp_path):
    """bfloat16 through the engine with CUDA graphs: every generated token is, for the plain model, the best token or within
    what rounding costs of it; and a captured step gives the tokens the same step gives when it is launched kernel by kernel."""
    d = make_model_dir("S", seed=3, root=str(tmp_path), sigma=0.2)
    cfg, w = read_model(d)
    prompts = [traces.make_requests(cfg["vocab"], [n], seed=n)["r0"] for n in (40, 3, 90, 9, 77)]
    eng = Engine(d, dtype="bfloat16", device=DEV, page_size=16, num_pages=40, num_slots=4)
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=12, ignore_eos=True))
    assert eng.runner.graph_steps > 0
    for p, o in zip(prompts, outs):
        toks = list(p) + o.token_ids
        lg = plain.forward(cfg, w, toks[:-1])
        slack = max(0.06 * float(lg.std()), 3 * rounding_cost(cfg, w, toks[:-1], lg))
        for i in range(len(p) - 1, len(toks) - 1):
            assert lg[i][toks[i + 1]] >= lg[i].max() - slack, (len(p), i)
    d = make_model_dir("V3", seed=3, root=str(tmp_path))
    prompts = [traces.make_requests(512, [n], seed=n)["r0"] for n in (40, 3, 90, 9)]
    tokens = []
    for graph in (True, False):
        eng = Engine(d, dtype="bfloat16", device=DEV, page_size=16, num_pages=60, num_slots=4, cuda_graph=graph)
        tokens.append([o.token_ids for o in eng.generate(prompts, SamplingParams(max_new_tokens=12, ignore_eos=True))])
        assert (eng.runner.graph_steps > 0) == graph
    assert tokens[0] == tokens[1]


# ------------------------------------------------------------------ the tools
def test_replay_tool_and_command_line(tmp_path_factory, tmp_path):
    d, cfg, w, reqs, oracle = model_and_oracle("V2", tmp_path_factory)
    steps = traces.mixed(reqs, seed=11)
    out_dir = str(tmp_path / "out")
    p = subprocess.Popen([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", out_dir, "--max-tokens",
                          str(traces.peak_tokens(steps))], stdin=subprocess.PIPE, stdout=subprocess.PIPE, text=True, cwd=ROOT)
    try:
        for s in steps:
            p.stdin.write(json.dumps(s) + "\n")
            p.stdin.flush()
            assert p.stdout.readline().strip() == f"done {s['step']}"
        p.stdin.close()
        assert p.wait(timeout=120) == 0
    finally:
        if p.poll() is None:
            p.kill()
    at = {r: 0 for r in reqs}
    for s in steps:
        rows = np.fromfile(os.path.join(out_dir, f"{s['step']}.f32"), dtype="<f4").reshape(-1, cfg["vocab"])
        k = 0
        for e in s["entries"]:
            n = len(e["want"])
            assert_close(torch.from_numpy(rows[k:k + n].copy()), oracle[e["id"]][at[e["id"]]: at[e["id"]] + n], torch.float32, e["id"])
            at[e["id"]] += n
            k += n
    ref = plain.generate_greedy(cfg, w, [5, 6, 7, 8], 6)
    r = subprocess.run([sys.executable, "-m", "arle_b200", "--model-path", d, "--dtype", "float32", "--max-tokens", "6", "--ignore-eos",
                        "--num-slots", "2", "--num-pages", "16", "run", "--prompt", "5 6 7 8", "--json"], capture_output=True, text=True, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(r.stdout)["outputs"][0]["token_ids"] == ref
