"""Tiny Dabilorn configurations for the tests.  Between them they vary every size and option of the design: the three mixers in
several orders and alone, layers without a feed-forward, experts with and without a shared expert, one chosen, several and all of
them, grouped, single and full key heads, values narrower, as wide and wider than keys, an odd head size, rotation of a part of a
head, of all of it and of none, stretched rotations (a ramp over several pairs, a ramp of no width, a factor of one, a factor below
one) and plain ones, chunks of one position, of a few (not a multiple of the page), of a page and longer than any test sequence, no
chunks at all, one to six convolution taps, memories of several sizes, and (D3) sizes that reach the kernels' wider paths."""
import json
import os
import tempfile

from arle_b200.weights import SafetensorsFile, write_random_model, write_safetensors


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base=10000.0, scaling=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": m}


def attn(heads, kv_heads, dim, vdim, scale, chunk=None, rot_dims=0, base=10000.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
    return {"type": "attention", "mixer": m}


def wkv(heads, dim, rank):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "decay_rank": rank}}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp):
    return json.loads(json.dumps({"type": mixer["type"], "mixer": mixer["mixer"], "mlp": mlp}))      # no two layers share an object


def model(vocab, width, eps, taps, layers):
    return {"architecture": "Dabilorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps}, "layers": layers}


TINY_D1 = model(211, 64, 1e-5, 4, [
    layer(latent(3, 8, 4, 12, 20, 28, 0.3, base=500.0, scaling=(4.0, 64, 8.0, 1.0)), moe(6, 2, 40, shared=24)),
    layer(attn(4, 2, 12, 20, 0.25, chunk=7, rot_dims=8, base=300.0), moe(5, 3, 16)),
    layer(wkv(3, 8, 5), moe(6, 1, 24, shared=48)),
    layer(attn(3, 1, 8, 8, 0.35, chunk=10, rot_dims=8), None)])
# D2: one tap (nothing to remember), sizes that other models make equal all different or all 1, a memory first, chunks of one
# position, no chunks, no rotation, an odd head size, a stretched rotation whose ramp has no width, factors of one and below one
TINY_D2 = model(157, 48, 2e-6, 1, [
    layer(wkv(1, 20, 9), moe(3, 3, 24)),
    layer(attn(6, 6, 9, 4, 0.4, chunk=1, rot_dims=6), moe(4, 1, 12, shared=8)),
    layer(latent(1, 24, 8, 16, 36, 40, 0.2, scaling=(1.0, 512, 4.0, 2.0)), None),
    layer(attn(1, 1, 12, 40, 0.3), moe(4, 4, 16)),
    layer(latent(5, 4, 6, 6, 44, 8, 0.5, base=90.0, scaling=(0.5, 3000, 1e6, 1e5)), moe(8, 5, 12, shared=20)),
    layer(wkv(5, 4, 30), None),
    layer(latent(2, 0, 12, 10, 12, 16, 0.4, base=1e6), moe(2, 1, 20))])
# D3: wider: heads of 64 and 128 with values as wide as keys, latents of 64 and 256, aligned rows, chunks of three pages and more
TINY_D3 = model(384, 192, 3e-6, 2, [
    layer(attn(8, 2, 64, 64, 0.125, chunk=48, rot_dims=32, base=50000.0), moe(16, 4, 96, shared=64)),
    layer(latent(8, 32, 32, 64, 64, 96, 0.17, base=20000.0, scaling=(8.0, 256, 16.0, 2.0)), moe(8, 2, 64)),
    layer(wkv(2, 64, 24), moe(8, 2, 64, shared=160)),
    layer(attn(4, 1, 128, 128, 0.09, chunk=200, rot_dims=128), None),
    layer(latent(4, 64, 16, 32, 256, 160, 0.125), None),
    layer(attn(2, 2, 128, 128, 0.09, rot_dims=64), moe(4, 1, 32))])
# A: the chunked attention alone, L: the latent attention alone, W: the memory alone (one number of taps each), for the tests that
# sharpen them; F: nothing gives pages back before a request ends
TINY_A = model(180, 64, 1e-5, 2, [layer(attn(2, 1, 16, 16, 0.25, chunk=6, rot_dims=8), None)])
TINY_L = model(180, 64, 1e-5, 3, [layer(latent(2, 16, 8, 8, 24, 16, 0.25, base=1000.0, scaling=(4.0, 32, 4.0, 0.5)), None)])
TINY_W = model(180, 64, 1e-5, 6, [layer(wkv(2, 16, 8), None), layer(wkv(4, 8, 12), moe(3, 2, 24, shared=16))])
TINY_F = model(180, 64, 1e-5, 3, [layer(attn(2, 2, 16, 12, 0.25, chunk=4000, rot_dims=16), moe(4, 2, 32, shared=16)),
                                  layer(wkv(2, 8, 4), None), layer(latent(2, 16, 8, 8, 24, 16, 0.25), None)])
CONFIGS = {"D1": TINY_D1, "D2": TINY_D2, "D3": TINY_D3, "A": TINY_A, "L": TINY_L, "W": TINY_W, "F": TINY_F}
INIT = {n: dict(sigma=0.12, gain_jitter=0.4) for n in CONFIGS}
INIT["D2"] = dict(sigma=0.14, gain_jitter=0.4)
INIT["D3"] = dict(sigma=0.07, gain_jitter=0.4)
PAGE_SIZES = {"D1": 4, "D2": 8, "D3": 16, "A": 4, "L": 4, "W": 8, "F": 16}


def make_model_dir(name: str, seed: int = 0, root: str = None, branches: float = 1.0, **init) -> str:
    """``branches``: every layer scale times this.  The output projection is the embedding table, so a model whose branches are
    no larger than its embedded token mostly repeats that token; larger branches make a greedy continuation wander."""
    root = root or tempfile.mkdtemp(prefix=f"arle_tiny_{name}_")
    kw = dict(INIT[name])
    kw.update(init)
    d = write_random_model(os.path.join(root, name), CONFIGS[name], seed, **kw)
    if branches != 1.0:
        change_tensors(d, lambda t: t.update({n: (v.float() * branches).to(v.dtype) for n, v in t.items() if ".ls" in n}))
    return d


def change_tensors(d: str, change) -> None:
    """``change`` gets the folder's tensors by name and alters the dict."""
    path = os.path.join(d, "model.safetensors")
    f = SafetensorsFile(path)
    t = {n: f.tensor(n).clone() for n in f.names()}
    change(t)
    write_safetensors(path, t)


def read_model(d: str):
    """(config dict, weights by name in float64) for the plain implementation."""
    import torch
    from safetensors.torch import load_file

    with open(os.path.join(d, "config.json")) as f:
        cfg = json.load(f)
    return cfg, {k: v.to(torch.float64) for k, v in load_file(os.path.join(d, "model.safetensors")).items()}
