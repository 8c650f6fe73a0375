"""Dabilorn on the GPU against the plain implementation (``plain_dabilorn``): every new or widened kernel alone at sizes of no
model (chunked attention with sigmoid weights in the general kernel and in the three tensor-core kernels, the row-wide norm with
values of their own width, interleaved and stretched rotation of latents, the layer norms, the input convolution and the token
shift continuing from states in permuted slots, the decay and the memory with a bonus, gates per number, experts weighted on their
input), the engine under every cutting in float32 and bfloat16 on tiny configurations, the first tokens of a sequence and prompts
that end on page and chunk borders, keys just inside and just outside a chunk made to decide the logits, a far key deciding them
through the latents (and through the stretched rotation), far tokens living on in the memories, the convolution's and the shift's
memories alone, long decoding while chunks' pages turn over, a request that starts again, greedy generation through the public
entry point with CUDA graphs and preemption, and the replay tool and the command line as subprocesses."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import kernel_refs
import plain_dabilorn as plain
import traces
from arle_b200 import Engine, ops
from arle_b200.engine import ModelRunner, StepEntry, load_model
from arle_b200.sampling import SamplingParams
from tiny_dabilorn import PAGE_SIZES, change_tensors, make_model_dir, read_model

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
LENGTHS = {"D1": [1, 5, 12, 23, 70, 130, 33], "D2": [2, 17, 40, 96, 64, 31], "D3": [3, 66, 150, 64, 40, 230], "W": [2, 33, 80, 17, 64],
           "A": [3, 50, 64, 29]}
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
    (a number: that argument; a string: that keyword's tensor)."""
    def on(a, dev):
        if isinstance(a, torch.Tensor):
            return a.to(dev) if dev else a.clone()
        if isinstance(a, tuple) and a and all(isinstance(x, torch.Tensor) or x is None for x in a):
            return tuple(on(x, dev) for x in a)
        return a
    kwargs = kwargs or {}
    cpu, gpu = [on(a, None) for a in args], [on(a, DEV) for a in args]
    ck, gk = {k: on(v, None) for k, v in kwargs.items()}, {k: on(v, DEV) for k, v in kwargs.items()}
    getattr(ops, fn)(*gpu, **gk)
    getattr(kernel_refs, fn)(*cpu, **ck)
    torch.cuda.synchronize()
    return [((gk[i] if isinstance(i, str) else gpu[i]), (ck[i] if isinstance(i, str) else cpu[i])) for i in outs]


def _close(pairs, dtype, **tol):
    for got, want in pairs:
        if isinstance(got, tuple):
            _close([(a, b) for a, b in zip(got, want) if a is not None], dtype, **tol)
        else:
            torch.testing.assert_close(got.float().cpu(), want.float(), **(tol or _tol(dtype)))


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


# ------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("nq,nkv,hd,vd,chunk,ps,sig", [(4, 2, 16, 24, 7, 4, True), (1, 1, 12, 40, 5, 8, True), (6, 2, 9, 4, 1, 16, True),
                                                       (3, 1, 48, 48, 33, 16, False), (2, 2, 80, 32, 0, 4, True), (5, 5, 20, 20, 40, 16, True)])
def test_chunked_attention_with_sigmoid_weights(dtype, nq, nkv, hd, vd, chunk, ps, sig):
    """The general kernel: rows that start at 0, inside a chunk, on a chunk's border and far on; the pages of passed chunks hold
    poison, so a kernel that looked there shows."""
    g = torch.Generator().manual_seed(hd + vd + chunk)
    starts, lens = [0, 2, 2 * chunk, 60, 119], [70, 9, 31, 1, 12]
    pages, bt, pos, row, slots, _ = _rows(g, starts, lens, ps)
    T = int(pos.numel())
    q = torch.randn(T, nq * hd, generator=g).to(dtype)
    kc = torch.randn(pages, nkv, ps, hd, generator=g).to(dtype)
    vc = torch.randn(pages, nkv, ps, vd, generator=g).to(dtype)
    if chunk:
        for r, s in enumerate(starts):
            for p in range((s // chunk * chunk) // ps):
                kc[bt[r, p]] = 1e4
                vc[bt[r, p]] = float("nan")
    out = torch.zeros(T, nq * vd, dtype=dtype)
    kw = dict(vd=vd, chunk=chunk or None, score_bias=torch.randn(nq, generator=g) - 2.0 if sig else None)
    (got, want), = _both("paged_attention", [q, out, kc, vc, pos, row, bt, nq, nkv, hd, ps, 0.3, None], [1], kw)
    assert torch.isfinite(got).all()
    _close([(got, want)], dtype)


@pytest.mark.parametrize("nq,nkv,hd,ps,chunk,window", [(8, 2, 128, 16, 37, None), (4, 1, 64, 16, 64, None), (2, 2, 64, 32, 300, None), (12, 4, 128, 8, 128, None),
                                                       (4, 2, 128, 16, None, None), (2, 1, 128, 32, 130, None), (4, 2, 128, 16, 5, None), (2, 2, 128, 16, 1000, None),
                                                       (2, 2, 128, 16, None, 45), (16, 1, 64, 16, 16, None), (2, 2, 64, 16, None, 7)])
def test_sigmoid_weights_and_chunks_in_the_tensor_core_attention_kernels(nq, nkv, hd, ps, chunk, window):
    """Prompts on mma.sync and on tcgen05 (chunks shorter than its 128-key tiles, as long, longer, and not a multiple; portions
    that start inside a chunk and on its border) and decoding with split keys (one split and several): each against the plain
    statement.  The pages that no query can see hold poison."""
    from test_kernels_gpu import _fast_setup

    scale = 4.0 / math.sqrt(hd)
    bias = torch.linspace(-4.0, 1.0, nq)

    def first(p):
        return p // chunk * chunk if chunk else max(0, p - window + 1) if window else 0

    def want(q, kc, vc, pos, rows, bt):
        exp = torch.empty(q.shape[0], nq * hd, dtype=torch.bfloat16)
        kernel_refs.paged_attention(q.cpu(), exp, kc.cpu(), vc.cpu(), pos.cpu(), rows.cpu(), bt.cpu(), nq, nkv, hd, ps, scale, window, chunk=chunk,
                                    score_bias=bias)
        return exp.float()

    def poison(kc, vc, bt, lens, q_lens):
        for r, (n, ql) in enumerate(zip(lens, q_lens)):
            for p in range(first(n - ql) // ps):
                kc[bt[r, p]] = 1e3
                vc[bt[r, p]] = float("nan")

    def close(out, exp, pos):
        # a weight is rounded to bfloat16 before the product with the values and nothing is divided by the weights' sum: the error
        # of a sum over n keys grows with the root of n (a key too many or too few moves it by that key's value)
        n = torch.tensor([int(p) - first(int(p)) + 1 for p in pos], dtype=torch.float32)
        err = (out.float().cpu() - exp).abs()
        tol = 0.01 + 0.006 * n.sqrt()[:, None] + 0.01 * exp.abs()
        assert (err <= tol).all(), f"token {int((err > tol).any(-1).nonzero()[0])}: error {float((err - tol).max()):.3g} above the tolerance"

    c = chunk or 100
    lens, q_lens = [130, 300, 128, 129, 9, 700, 2 * c + 3], [130, 2, 128, 3, 1, 333, 3]
    q, kc, vc, pos, rows, bt, qi, kv = _fast_setup(nq, nkv, hd, ps, lens, q_lens, seed=6)
    poison(kc, vc, bt, lens, q_lens)
    exp = want(q, kc, vc, pos, rows, bt)
    for fn in ([ops.paged_attention_prefill_tc] if hd == 128 and ps % 16 == 0 else []) + [ops.paged_attention_prefill]:
        out = torch.zeros(q.shape[0], nq * hd, dtype=torch.bfloat16, device=DEV)
        fn(q, out, kc, vc, qi, kv, bt, nq, nkv, hd, ps, scale, window, max(q_lens), chunk=chunk or 0, score_bias=bias.to(DEV))
        ops.check_errors(DEV)
        close(out, exp, pos)
    lens = [1, 63, 64, 65, 700, 2049, 17, c, c + 1, 2 * c, 3 * c - 1]
    R = len(lens)
    q, kc, vc, pos, rows, bt, qi, kv = _fast_setup(nq, nkv, hd, ps, lens, [1] * R, seed=3)
    poison(kc, vc, bt, lens, [1] * R)
    exp = want(q, kc, vc, pos, rows, bt)
    for splits in (1, 2, 5):
        out = torch.zeros(R, nq * hd, dtype=torch.bfloat16, device=DEV)
        po, pml = torch.zeros(R * nq * splits * hd, device=DEV), torch.zeros(R * nq * splits * 2, device=DEV)
        ops.paged_attention_decode(q, out, kc, vc, qi, kv, bt, nq, nkv, hd, ps, scale, window, splits, po, pml,
                                   torch.zeros(R * nkv, dtype=torch.int32, device=DEV), chunk=chunk or 0, score_bias=bias.to(DEV))
        close(out, exp, pos)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("nq,nkv,hd,vd,rdim,ps", [(4, 2, 16, 24, 8, 4), (1, 1, 12, 40, 12, 8), (6, 3, 9, 5, 6, 16), (3, 1, 48, 20, 48, 16), (2, 1, 130, 64, 0, 16),
                                                  (8, 4, 64, 32, 64, 32)])
def test_preparation_with_the_norm_over_the_row_and_values_of_their_own_width(dtype, nq, nkv, hd, vd, rdim, ps):
    g = torch.Generator().manual_seed(hd)
    pages, bt, pos, row, slots, _ = _rows(g, [0, 13, 200], [9, 4, 1], ps)
    T, n = int(pos.numel()), nq * hd + nkv * (hd + vd)
    qkv = torch.randn(T, n + 3, generator=g).to(dtype)[:, :n]
    wq, wk = (torch.rand(m * hd, generator=g) + 0.5 for m in (nq, nkv))
    inv = torch.pow(torch.tensor(300.0), -torch.arange(rdim // 2) * 2.0 / max(rdim, 1)).float()
    kc, vc = torch.zeros(pages, nkv, ps, hd, dtype=dtype), torch.zeros(pages, nkv, ps, vd, dtype=dtype)
    args = [qkv, pos, slots, wq, wk, 1e-5, inv if rdim else None, rdim, "half", False, kc, vc, nq, nkv, hd, ps]
    _close(_both("attention_prep_row", args, [0, 10, 11], dict(vd=vd)), dtype)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("H,dn,dr,rank,rdim,pairing,amp", [(3, 8, 4, 20, 4, "interleaved", 1.2), (1, 0, 12, 36, 12, "interleaved", 1.0), (8, 32, 32, 64, 16, "half", 0.9),
                                                           (5, 4, 6, 44, 6, "interleaved", 1.4), (2, 16, 64, 128, 64, "half", 1.0)])
def test_latent_preparation_with_either_pairing_and_an_amplitude(dtype, H, dn, dr, rank, rdim, pairing, amp):
    g = torch.Generator().manual_seed(rank)
    ps = 8
    pages, bt, pos, row, slots, _ = _rows(g, [0, 13, 900], [9, 4, 1], ps)
    T = int(pos.numel())
    q = torch.randn(T, H * (dn + dr) + 2, generator=g).to(dtype)[:, : H * (dn + dr)]
    dkv = torch.randn(T, rank + dr + 4, generator=g).to(dtype)[:, 2: rank + dr + 2]
    inv = torch.pow(torch.tensor(500.0), -torch.arange(rdim // 2) * 2.0 / rdim).float()
    cache, q_abs = torch.zeros(pages, 1, ps, rank + dr, dtype=dtype), torch.zeros(T, H, rank + dr, dtype=dtype)
    args = [q, dkv, pos, slots, torch.rand(rank, generator=g) + 0.5, 1e-5, inv, rdim, cache, q_abs, H, dn, dr, rank]
    tol = dict(rtol=1e-4, atol=2e-4) if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)      # angles of 900 radians
    _close(_both("latent_prep", args, [8, 9], dict(pairing=pairing, amplitude=amp)), dtype, **tol)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("T,H", [(1, 48), (7, 64), (33, 1000), (3, 4096), (5, 130), (2, 9001)])
def test_layer_norms(dtype, T, H):
    """Rows with a mean far from zero: the variance is that of the deviations."""
    g = torch.Generator().manual_seed(H)
    resid = torch.randn(T, H, generator=g) * 3 + 20.0
    delta = torch.randn(T, H, generator=g).to(dtype)
    w = torch.rand(H, generator=g) + 0.5
    rows = torch.randperm(T, generator=g)[: max(1, T // 2)].to(torch.int32)
    tol = dict(rtol=2e-5, atol=5e-5) if dtype == torch.float32 else _tol(dtype)
    _close(_both("layernorm", [resid, None, None, w, 1e-5, torch.zeros(T, H, dtype=dtype), False], [5]), dtype, **tol)
    _close(_both("layernorm", [resid, delta, None, w, 2e-6, torch.zeros(T, H, dtype=dtype), True], [0, 5]), dtype, **tol)
    _close(_both("layernorm", [resid, delta, rows, w, 1e-5, torch.zeros(len(rows), H, dtype=dtype), False], [0, 5]), dtype, **tol)
    in_place = resid.to(DEV)
    ops.layernorm(in_place, None, None, w.to(DEV), 1e-5, in_place, False)
    want = torch.zeros(T, H)
    kernel_refs.layernorm(resid, None, None, w, 1e-5, want, False)
    torch.testing.assert_close(in_place.cpu(), want, rtol=2e-5, atol=5e-5)
    branch = (torch.randn(T, H + 8, generator=g) * 0.2 - 1.0).to(dtype)[:, :H]
    _close(_both("branch_layernorm_add", [resid, branch, w, 1e-5, torch.zeros(T, H, dtype=dtype)], [0, 4]), dtype, **tol)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("C,taps,lens", [(48, 4, [1, 5, 40]), (64, 2, [18, 1, 2]), (130, 3, [33, 1, 9]), (256, 6, [1, 1, 1]), (96, 1, [7, 1]), (20, 9, [3, 20, 1]),
                                         (1024, 3, [1, 1])])
def test_input_convolution_and_token_shift(dtype, C, taps, lens):
    """Rows of unequal length that continue from memories in permuted slots, shorter and longer than what is remembered."""
    g = torch.Generator().manual_seed(C + taps)
    T, R = sum(lens), len(lens)
    slots = torch.randperm(R + 2, generator=g)[:R].to(torch.int32)
    indptr = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32)
    row = torch.cat([torch.full((n,), r) for r, n in enumerate(lens)]).to(torch.int32)
    n = C * (taps - 1)
    x, w = torch.randn(T, C, generator=g), torch.randn(taps, C, generator=g)
    for pad in (0, 3):                                      # slots on 16-byte boundaries, and not
        state = torch.randn(R + 2, max(n, 1) + 4 + pad, generator=g)
        _close(_both("input_conv", [x, w, state, indptr, row, slots, torch.zeros(T, C, dtype=dtype), max(lens)], [2, 6]), dtype)
        mu = torch.rand(5, C, generator=g)
        h = torch.randn(T, C + 8, generator=g).to(dtype)[:, 4: C + 4]
        state = torch.randn(R + 2, C + 4 + pad, generator=g)
        _close(_both("token_shift", [h, mu, state, indptr, row, slots, torch.zeros(5, T, C, dtype=dtype), max(lens)], [2, 6]), dtype)
        if max(lens) == 1:                                  # the convolution inside the kernel that ends the block before
            branch = torch.randn(T, C, generator=g).to(dtype)
            state = torch.randn(R + 2, max(n, 1) + 4 + pad, generator=g)
            args = [x, branch, torch.rand(C, generator=g) + 0.5, 1e-5, None]
            _close(_both("branch_layernorm_add", args, [0, "conv"], dict(conv=(w, state, slots, torch.zeros(T, C, dtype=dtype)))), dtype,
                   **(dict(rtol=1e-4, atol=1e-4) if dtype == torch.float32 else dict(rtol=2e-2, atol=5e-2)))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("H,D,rank,lens", [(3, 8, 5, [1, 5, 40]), (1, 20, 9, [18, 1, 2]), (4, 64, 24, [33, 1, 9]), (5, 4, 30, [1, 1, 1]), (2, 160, 700, [70, 3]),
                                           (4, 32, 16, [300]), (2, 128, 64, [2, 65]), (1, 300, 8, [9, 1])])
def test_decay_and_memory_with_a_bonus(dtype, H, D, rank, lens):
    g = torch.Generator().manual_seed(D)
    T, R, N = sum(lens), len(lens), H * D
    low = torch.randn(T, rank, generator=g)
    w2 = torch.randn(rank, N, generator=g) * rank ** -0.5
    bias = torch.randn(N, generator=g) * 2 - 2
    decay = torch.zeros(T, N)
    _close(_both("gla_decay", [low, w2, bias, 1.0, decay], [4], dict(form="double_exp")), torch.float32, rtol=1e-4, atol=1e-5)
    kernel_refs.gla_decay(low, w2, bias, 1.0, decay, form="double_exp")
    r, k, v = (torch.randn(T, N, generator=g).to(dtype) for _ in range(3))
    bonus = torch.randn(N, generator=g)
    slots = torch.randperm(R + 2, generator=g)[:R].to(torch.int32)
    indptr = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32)
    tol = dict(rtol=2e-4, atol=2e-3) if dtype == torch.float32 else dict(rtol=2e-2, atol=5e-2)
    for pad in (4, 7):
        state = torch.randn(R + 2, N * D + pad, generator=g) * 0.5
        args = [r, k, v, decay, state, indptr, slots, torch.zeros(T, N), H, D, D, 1.0, max(lens)]
        _close(_both("gla_scan", args, [4, 7], dict(bonus=bonus)), dtype, **tol)
    o, wt = torch.randn(T, N, generator=g), torch.rand(N, generator=g) + 0.5
    gate = torch.randn(T, N, generator=g).to(dtype)
    _close(_both("gla_out", [o, gate, wt, 1e-5, 1.0, torch.zeros(T, N, dtype=dtype), H, D], [5]), dtype)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_gates_per_number_and_the_square_of_relu(dtype):
    g = torch.Generator().manual_seed(3)
    for T, n in ((5, 36), (3, 128), (70, 1000), (2, 4101)):
        x = torch.randn(T, n + 8, generator=g).to(dtype)[:, 8:]
        gate = torch.randn(T, n + 16, generator=g).to(dtype)[:, 8: n + 8] * 3
        _close(_both("gate_mul", [x, gate, torch.zeros(T, n, dtype=dtype)], [2]), dtype)
        _close(_both("square_relu", [x, torch.zeros(T, n, dtype=dtype)], [1]), dtype)
    for M, K, N in ((1, 64, 40), (8, 4096, 136), (5, 8192, 24), (30, 96, 64), (3, 20, 12)):         # one CTA's sums, a cluster's, many rows
        x, w = torch.randn(M, K, generator=g).to(dtype), (torch.randn(N, K, generator=g) * K ** -0.5).to(dtype)
        _close(_both("gemm_square_relu", [x, w, torch.zeros(M, N, dtype=dtype)], [2]), dtype)
    for M, heads, K, N in ((7, 3, 24, 20), (130, 4, 64, 32), (5, 2, 9, 11), (70, 2, 256, 136)):
        x = torch.randn(M, heads, K, generator=g).to(dtype)
        w = (torch.randn(heads, N, K, generator=g) * K ** -0.5).to(dtype)
        gate = torch.randn(M, heads * N + 8, generator=g).to(dtype)[:, 8:]
        _close(_both("gemm_heads", [x, w, torch.zeros(M, heads, N, dtype=dtype)], [2], dict(gate=gate)), dtype)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("T,E,top,K,N", [(9, 12, 2, 48, 40), (70, 5, 5, 64, 96), (3, 64, 1, 20, 12), (130, 7, 3, 256, 136), (300, 9, 4, 128, 64)])
def test_experts_weighted_on_their_input(dtype, T, E, top, K, N):
    """The grouped product with a number per place and the square of relu on its sums, against w applied to the rows first."""
    g = torch.Generator().manual_seed(T)
    x = torch.randn(T, K, generator=g).to(dtype)
    w = (torch.randn(E, N, K, generator=g) * K ** -0.5).to(dtype)
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    wts = torch.rand(T, top, generator=g) + 0.1
    pairs = T * top
    plan = torch.zeros(ops.moe_plan_size(E, pairs), dtype=torch.int32, device=DEV)
    place, row, of_place = (torch.zeros(pairs, dtype=d, device=DEV) for d in (torch.int32, torch.int32, torch.float32))
    ops.moe_plan(ids.to(DEV), E, plan, place, row, wts.to(DEV), of_place)
    assert torch.equal(of_place.cpu()[place.cpu().long()], wts.reshape(-1))
    out, y = torch.zeros(pairs, N, dtype=dtype, device=DEV), torch.zeros(T, N, dtype=dtype, device=DEV)
    ops.moe_gemm(x.to(DEV), row, w.to(DEV), out, plan, E, place_scale=of_place, act="square_relu")
    xw = (x.float()[:, None, :] * wts[:, :, None]).reshape(pairs, K)
    want = torch.einsum("pk,pnk->pn", xw, w.float()[ids.reshape(-1).long()]).clamp(min=0.0) ** 2
    torch.testing.assert_close(out.float().cpu()[place.cpu().long()], want, **_tol(dtype))
    shared, gate = torch.randn(T, N, generator=g).to(dtype), torch.randn(T, generator=g)
    ops.moe_combine(out, place, None, shared.to(DEV), gate.to(DEV), y, top=top)
    total = want.view(T, top, N).sum(1) + torch.sigmoid(gate)[:, None] * shared.float()
    torch.testing.assert_close(y.float().cpu(), total, **(_tol(dtype) if dtype == torch.float32 else dict(rtol=3e-2, atol=6e-2)))


# ------------------------------------------------------------------ the engine under every cutting
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("cut", ["whole", "tail_decode", "portions", "mixed"])
@pytest.mark.parametrize("name", ["D1", "D2", "D3", "W"])
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
    d, cfg, w, reqs, oracle = model_and_oracle("D3", tmp_path_factory)
    steps = traces.mixed(reqs, seed=9)
    for ps, ks in ((32, "fast"), (64, "fast"), (16, "plain")):
        runner = ModelRunner(load_model(d, dtype, DEV), ps, max(1, -(-traces.peak_tokens(steps) // ps)), 4, device=DEV, kernel_set=ks)
        got = traces.run_trace(runner, steps)
        for r, want in oracle.items():
            assert_close(got[r], want, dtype, f"pages of {ps}, {ks} kernels, request {r}", _rounding[id(oracle)])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", ["D1", "D2", "W"])
def test_first_tokens_page_and_chunk_borders(name, dtype, tmp_path_factory):
    d, cfg, w, reqs, oracle = model_and_oracle(name, tmp_path_factory)
    ps = PAGE_SIZES[name]
    runner = ModelRunner(load_model(d, dtype, DEV), ps, 64, 3, device=DEV)
    toks = [7, 7, 3, 150, 1, 9, 9]
    want = plain.forward(cfg, w, toks)
    rc = _rounding[id(oracle)]
    one_by_one = torch.cat([runner.step([StepEntry("a", [t], (0,))]).clone() for t in toks])
    together = runner.step([StepEntry("b", toks, range(7))]).clone()
    assert_close(one_by_one, want, dtype, "one by one", rc)
    assert_close(together, want, dtype, "together", rc)
    runner.end_request("a"), runner.end_request("b")
    # prompts that end exactly on a page's or a chunk's border, one before and one after, then two decoded tokens
    long = traces.make_requests(cfg["vocab"], [4 * ps + 3], seed=2)["r0"]
    want = plain.forward(cfg, w, long)
    for n in (ps - 1, ps, ps + 1, 2 * ps, 4 * ps, 6, 7, 9, 10, 14):
        got = [runner.step([StepEntry("c", long[:n], range(n))]).clone()]
        got += [runner.step([StepEntry("c", [long[n + i]], (0,))]).clone() for i in range(2)]
        assert_close(torch.cat(got), want[: n + 2], dtype, f"prompt of {n}", rc)
        runner.end_request("c")


def _changed(name, tmp_path, change, length, edit_config=None):
    """A tiny model with some tensors (and configuration values) changed: (folder, config, weights, tokens, the plain logits,
    what rounding costs)."""
    d = make_model_dir(name, seed=9, root=str(tmp_path))
    change_tensors(d, change)
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
def test_keys_at_the_chunks_edges_and_the_score_bias_decide_the_logits(dtype, tmp_path):
    """Random weights make the scores small and the weights nearly equal.  The score scale and the layer scale are raised until
    single keys count.  The plain model with chunks one longer or one shorter, with chunks that start one position later, or
    without the number added to the scores is far from the plain model at several positions, so such a fault would show; the
    engine is not, in prompts cut at every kind of place and in decoding."""
    d, cfg, w, toks, want, rc = _changed("A", tmp_path, lambda t: (_scale(t, "l0.ls1", 3.0), _scale(t, "l0.mix.pb", 4.0)), 90,
                                         lambda cfg: cfg["layers"][0]["mixer"].update(scale=1.5))
    tol = max(REL[dtype] * float(want.std()), 4.5 * rc if dtype == torch.bfloat16 else 0.0)

    def shows(logits, what):
        wrong = (logits - want).abs().max(dim=-1).values
        assert (wrong > 3 * tol).sum() >= 2, f"{what} would not show"

    for delta in (1, -1):
        off = copy.deepcopy(cfg)
        off["layers"][0]["mixer"]["mask"]["size"] += delta
        shows(plain.forward(off, w, toks), f"chunks off by {delta}")
    usual = plain.causal
    try:
        plain.causal = lambda T, chunk=None: usual(T + 1, chunk)[1:, 1:]        # chunks counted from position -1
        shows(plain.forward(cfg, w, toks), "chunks that start elsewhere")
        plain.causal = lambda T, chunk=None: usual(T)                           # no chunks
        shows(plain.forward(cfg, w, toks), "no chunks")
    finally:
        plain.causal = usual
    shows(plain.forward(cfg, dict(w, **{"l0.mix.pb": torch.zeros_like(w["l0.mix.pb"])}), toks), "scores without their number")
    for sizes in CUTS_90:
        assert_close(_run_cut(d, dtype, PAGE_SIZES["A"], toks, sizes), want, dtype, f"cut {sizes[:4]}", rc)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_a_far_key_decides_the_logits_through_the_latents(dtype, tmp_path):
    """A latent attention that sees every earlier token, sharpened, 330 tokens over many pages: late logits depend on single far
    tokens; and they depend on the stretched frequencies, on the amplitude and on the pairing of the rotated numbers."""
    d, cfg, w, toks, want, rc = _changed("L", tmp_path, lambda t: _scale(t, "l0.ls1", 3.0), 330, lambda cfg: cfg["layers"][0]["mixer"].update(scale=0.5))
    tol = max(REL[dtype] * float(want.std()), 4.5 * rc if dtype == torch.bfloat16 else 0.0)
    moved = list(toks)
    moved[5] = (moved[5] + 1) % cfg["vocab"]
    effect = (plain.forward(cfg, w, moved)[200:] - want[200:]).abs().max().item() / float(want.std())
    assert effect > 1e-2, "the sharpened layer does not look far back"
    usual_rotate, usual_stretch = plain.rotate, plain.stretched_frequencies
    try:
        for what, rot, stretch in (("half-split pairs", lambda x, p, f, i, a=1.0: usual_rotate(x, p, f, False, a), usual_stretch),
                                   ("no amplitude", lambda x, p, f, i, a=1.0: usual_rotate(x, p, f, i), usual_stretch),
                                   ("frequencies as they are", usual_rotate, lambda b, n, *k: (plain.frequencies(b, n), usual_stretch(b, n, *k)[1]))):
            plain.rotate, plain.stretched_frequencies = rot, stretch
            wrong = (plain.forward(cfg, w, toks) - want).abs().max(dim=-1).values
            assert (wrong > 3 * tol).sum() >= 5, f"{what} would not show"
    finally:
        plain.rotate, plain.stretched_frequencies = usual_rotate, usual_stretch
    assert_close(_run_cut(d, dtype, PAGE_SIZES["L"], toks, (130, 1, 1, 64, 2, 99, 1, 1) + (1,) * 31), want, dtype, "far", rc)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_a_far_token_lives_on_in_the_memories(dtype, tmp_path):
    """Decays next to one (w0 far below zero): the memories keep what the first tokens wrote for hundreds of steps, and a memory
    that is lost, reset or mixed up between steps shows; so does a bonus that is left out."""
    def change(t):
        for l in (0, 1):
            t[f"l{l}.mix.w0"] = (t[f"l{l}.mix.w0"].float() - 7.0).to(torch.bfloat16)
            _scale(t, f"l{l}.ls1", 3.0)
            _scale(t, f"l{l}.mix.u", 4.0)
    d, cfg, w, toks, want, rc = _changed("W", tmp_path, change, 250)
    moved = list(toks)
    moved[5] = (moved[5] + 1) % cfg["vocab"]
    effect = (plain.forward(cfg, w, moved)[200:] - want[200:]).abs().max().item() / float(want.std())
    assert effect > 1e-2, "the memories do not remember far tokens"
    none = dict(w, **{f"l{l}.mix.u": torch.zeros_like(w[f"l{l}.mix.u"]) for l in (0, 1)})
    assert (plain.forward(cfg, none, toks) - want).abs().max() > 0.1 * float(want.std())
    assert_close(_run_cut(d, dtype, PAGE_SIZES["W"], toks, (100, 1, 1, 64, 2, 49, 1, 1) + (1,) * 31), want, dtype, "state", rc)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_the_convolutions_and_the_shifts_memories(dtype, tmp_path):
    """Convolution weights and mixes raised: portions of two and three tokens (fewer than the six taps remember) and single tokens
    live on what earlier steps left."""
    def change(t):
        for l in (0, 1):
            _scale(t, f"l{l}.canon1", 3.0)
            _scale(t, f"l{l}.ls1", 2.0)
            for m in "rkvgw":
                _scale(t, f"l{l}.mix.mu.{m}", 3.0)
    d, cfg, w, toks, want, rc = _changed("W", tmp_path, change, 40)
    # without what earlier steps left, a portion would start like a sequence
    assert (plain.forward(cfg, w, toks[20:]) - want[20:]).abs().max(dim=-1).values[:3].min() > 0.05 * float(want.std())
    for sizes in ((40,), (2,) * 20, (3, 2, 1, 1, 4, 2, 5, 6, 7, 9), (1,) * 40, (20, 20)):
        assert_close(_run_cut(d, dtype, PAGE_SIZES["W"], toks, sizes), want, dtype, f"cut {sizes[:4]}", rc)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_long_decoding_keeps_cache_and_states_exact(dtype, tmp_path_factory):
    d, cfg, w, reqs, oracle = model_and_oracle("D1", tmp_path_factory)
    toks = traces.make_requests(cfg["vocab"], [320], seed=8)["r0"]
    want = plain.forward(cfg, w, toks)
    runner = ModelRunner(load_model(d, dtype, DEV), 4, 80, 2, device=DEV)         # pages of four: the chunks' pages turn over
    got = [runner.step([StepEntry("r", toks[:20], range(20))]).clone()]
    got += [runner.step([StepEntry("r", [t], (0,))]).clone() for t in toks[20:]]
    held = [g.pool.num_pages - g.pool.num_free for g in runner.cache.groups]
    assert held == [80, 2, 0]                    # every latent; 320 = 45 * 7 + 5: pages from 312 on; 320 = 32 * 10: nothing
    assert_close(torch.cat(got), want, dtype, "300 decoded tokens", rounding_cost(cfg, w, toks, want))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", ["W", "D1"])
def test_a_request_that_starts_again(name, dtype, tmp_path_factory):
    d, cfg, w, reqs, oracle = model_and_oracle(name, tmp_path_factory)
    steps = traces.preempted(reqs)
    ps = PAGE_SIZES[name]
    runner = ModelRunner(load_model(d, dtype, DEV), ps, traces.peak_tokens(steps) // ps, 3, device=DEV)
    for rid, pos, row in traces.run_trace_by_position(runner, steps):
        assert_close(row[None], oracle[rid][pos][None], dtype, f"{rid} at {pos}", _rounding[id(oracle)])


# ------------------------------------------------------------------ generation
@pytest.mark.parametrize("graph", [True, False], ids=["graphs", "eager"])
@pytest.mark.parametrize("name", ["F", "D1", "W", "D2"])
def test_greedy_generation_equals_plain_model_f32(name, graph, tmp_path):
    d = make_model_dir(name, seed=3, root=str(tmp_path), branches=4.0)
    cfg, w = read_model(d)
    prompts = [[5, 17, 3, 150, 9, 1, 1, 44, 102, 7, 7], [42] * 19, [7], list(range(20, 61))]
    ref = [plain.generate_greedy(cfg, w, p, 12) for p in prompts]
    assert all(len(set(r)) >= 3 for r in ref), "the continuation is too uniform to test anything"
    ps = PAGE_SIZES[name]
    for pages in (256 // ps, 112 // ps):                     # plenty; and so few that a request is preempted
        eng = Engine(d, dtype="float32", device=DEV, page_size=ps, num_pages=pages, num_slots=3, chunked_prefill_size=16,
                     max_num_batched_tokens=32, cuda_graph=graph)
        outs = eng.generate(prompts, SamplingParams(max_new_tokens=12, ignore_eos=True))
        assert [o.token_ids for o in outs] == ref, f"{pages} pages"
        assert not graph or eng.runner.graph_steps > 0
        eng.runner.cache.check()


def test_greedy_generation_bf16_stays_on_the_plain_models_best(tmp_path):
    """bfloat16 through the engine with CUDA graphs: every generated token is, for the plain model, the best token or within
    what rounding costs of it; and a captured step gives the tokens the same step gives when it is launched kernel by kernel."""
    d = make_model_dir("W", seed=3, root=str(tmp_path), branches=3.0)
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
    d = make_model_dir("D3", seed=3, root=str(tmp_path), branches=3.0)
    prompts = [traces.make_requests(384, [n], seed=n)["r0"] for n in (40, 3, 90, 9)]
    tokens = []
    for graph in (True, False):
        eng = Engine(d, dtype="bfloat16", device=DEV, page_size=16, num_pages=40, num_slots=4, cuda_graph=graph)
        tokens.append([o.token_ids for o in eng.generate(prompts, SamplingParams(max_new_tokens=12, ignore_eos=True))])
        assert (eng.runner.graph_steps > 0) == graph
    assert tokens[0] == tokens[1]


# ------------------------------------------------------------------ the tools
def test_replay_tool_and_command_line(tmp_path_factory, tmp_path):
    d, cfg, w, reqs, oracle = model_and_oracle("D2", tmp_path_factory)
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
