"""Tiny Virorax configurations for the tests.  Between them they vary every size and option of the design: the two mixers in
several orders (a retention layer first, one kind alone), layers with and without a feed-forward of either kind, loops over one
layer, several, all of them, that start at the first layer, end with the last, run once, twice, three and four times, and none;
grouped, single and full key heads, rotation of a part of a head, of all of it and of none, value widths below, at and above
the key width, an odd head size, windows of one token, of a few (not a multiple of the page), longer than any test sequence and
none, one memory and several with decays from 0 to 1, memories wider than long and longer than wide, a factor on the branches
below, at and above one, with and without capped logits, and (V3) sizes that reach the kernels' wider paths."""
import json
import os
import tempfile

from arle_b200.weights import write_random_model


def attn(heads, kv_heads, dim, vdim, scale, window=None, rot_dims=0, base=10000.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
    return {"type": "attention", "mixer": m}


def ret(heads, dim, vdim, decay, rot_dims=0, base=10000.0):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
    return {"type": "retention", "mixer": m}


def layer(mixer, ff=None):
    return json.loads(json.dumps({"type": mixer["type"], "mixer": mixer["mixer"], "mlp": {"kind": "dense", "ff": ff} if ff else None}))


def model(vocab, width, eps, mult, layers, loop=None, cap=None, positions=512):
    m = {"architecture": "Virorax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers,
         "max_positions": positions}
    if loop is not None:
        m["loop"] = dict(zip(("start", "stop", "times"), loop))
    if cap is not None:
        m["logit_softcap"] = cap
    return m


TINY_V1 = model(211, 64, 1e-5, 0.45, [
    layer(attn(4, 2, 16, 24, 0.3, window=7, rot_dims=8), 40),
    layer(ret(3, 8, 12, (0.6, 0.9, 0.999), rot_dims=4), None),
    layer(attn(2, 1, 12, 12, 0.2, window=11, rot_dims=12, base=900.0), 56),
    layer(ret(2, 16, 8, (0.97, 0.8), rot_dims=16), 24)], loop=(1, 3, 2), cap=9.0)
# V2: a retention layer first, a loop over everything, odd and unequal sizes, no window, no rotation, decays of 0 and 1, a
# factor of one on the branches, no cap
TINY_V2 = model(157, 48, 2e-6, 1.0, [
    layer(ret(1, 20, 8, (1.0,)), 20),
    layer(attn(6, 6, 8, 4, 0.4, window=1), None),
    layer(attn(6, 2, 9, 20, 0.5, rot_dims=6, base=500.0), 33),
    layer(ret(5, 4, 6, (0.0, 0.3, 0.5, 0.95, 1.0), rot_dims=2), None)], loop=(0, 4, 3), positions=700)
# V3: wider: heads of 64 and 128 with values as wide as keys, rotation of a half, a quarter and all of a head, memories of 128
TINY_V3 = model(512, 192, 3e-6, 0.8, [
    layer(ret(2, 128, 128, (0.9, 0.995), rot_dims=64, base=50000.0), 96),
    layer(attn(8, 2, 64, 64, 0.125, window=48, rot_dims=16, base=50000.0), 160),
    layer(attn(4, 1, 128, 128, 0.09, window=37, rot_dims=128), None),
    layer(ret(4, 64, 32, (0.7, 0.97, 0.999, 0.9), rot_dims=64), None),
    layer(attn(2, 2, 128, 128, 0.1, rot_dims=64), 128)], loop=(3, 5, 2), cap=20.0)
# A: attention alone (windows of 6 and 9) and R: retention alone, for the tests that sharpen them; F: windows longer than any
# test sequence; L: one layer looped four times; S: the memories with little else
TINY_A = model(180, 64, 1e-5, 0.9, [layer(attn(2, 1, 16, 16, 0.25, window=6, rot_dims=8), 32)])
TINY_R = model(180, 64, 1e-5, 0.9, [layer(ret(2, 16, 12, (0.999, 1.0), rot_dims=8), 24), layer(ret(3, 8, 4, (0.5, 0.9, 0.99)), None)])
TINY_F = model(180, 64, 1e-5, 1.3, [layer(attn(2, 2, 16, 12, 0.25, window=4000, rot_dims=16), 32), layer(attn(4, 2, 8, 8, 0.3, rot_dims=4), None)],
               loop=(1, 2, 2), cap=12.0)
TINY_L = model(180, 64, 1e-5, 0.5, [layer(attn(2, 1, 16, 16, 0.25, window=5, rot_dims=8), 32)], loop=(0, 1, 4))
TINY_S = model(180, 64, 1e-5, 0.9, [layer(attn(2, 1, 8, 8, 0.3, window=5, rot_dims=8), None), layer(ret(2, 16, 12, (0.999, 1.0), rot_dims=16), 24)],
               loop=(0, 2, 2), cap=15.0)
CONFIGS = {"V1": TINY_V1, "V2": TINY_V2, "V3": TINY_V3, "A": TINY_A, "R": TINY_R, "F": TINY_F, "L": TINY_L, "S": TINY_S}
INIT = {"V1": dict(sigma=0.12, gain_jitter=0.3), "V2": dict(sigma=0.14, gain_jitter=0.3), "V3": dict(sigma=0.07, gain_jitter=0.3)}
PAGE_SIZES = {"V1": 4, "V2": 8, "V3": 16, "A": 4, "R": 8, "F": 4, "L": 4, "S": 8}


def make_model_dir(name: str, seed: int = 0, root: str = None, **init) -> str:
    root = root or tempfile.mkdtemp(prefix=f"arle_tiny_{name}_")
    kw = dict(INIT.get(name, dict(sigma=0.12, gain_jitter=0.3)))
    kw.update(init)
    return write_random_model(os.path.join(root, name), CONFIGS[name], seed, **kw)


def read_model(d: str):
    """(config dict, weights by name in float64) for the plain implementation."""
    import torch
    from safetensors.torch import load_file

    with open(os.path.join(d, "config.json")) as f:
        cfg = json.load(f)
    return cfg, {k: v.to(torch.float64) for k, v in load_file(os.path.join(d, "model.safetensors")).items()}
