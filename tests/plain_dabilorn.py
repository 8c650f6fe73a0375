"""A plain, slow implementation of the Dabilorn design: float64 torch on the CPU, whole sequences,
no cache, no batching, one function per mechanism.  It shares no code with the package's model
path; the tests compare the engine with it.

A model is (config dict in the form of config.json, {tensor name: tensor}).  ``forward`` returns
the logits of every position and, on request, the residual after every layer.  ``rnd`` is applied to
every stored activation (identity by default; rounding to bfloat16 gives the tests the size of what
rounding alone does).

With LN a layer norm without bias, s1 and s2 two stored vectors and C a causal convolution per channel:
    x <- x + s1 * LN1(mixer(x + C x)),   x <- x + s2 * LN2(experts(x)).
Notation: h is a sublayer's input [T, width]; positions count from 0.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def _ident(x):
    return x


def round_bf16(x):
    return x.to(torch.float32).to(torch.bfloat16).to(F64)


def lin(W, x):
    """Rows of x through a matrix stored [out, in]."""
    return x @ W.to(F64).t()


# ----------------------------------------------------------------------------- small functions
def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w.to(F64)


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def plus_short_conv(h, w):
    """h [T, C], w [C, taps]: h_t + sum_j w[:, j] * h_(t - taps + 1 + j), zeros before the start."""
    T, taps = h.shape[0], w.shape[1]
    w = w.to(F64)
    y = h.clone()
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] = y[t] + w[:, j] * h[s]
    return y


def frequencies(base, dims):
    i = torch.arange(dims // 2, dtype=F64)
    return torch.pow(torch.tensor(float(base), dtype=F64), -2.0 * i / dims)


def stretched_frequencies(base, dims, factor, original, fast, slow):
    """Frequencies for a context ``factor`` times the original one: pairs that turn more than ``fast`` times within the
    original context keep theirs, pairs that turn fewer than ``slow`` times are divided by the factor, a linear ramp
    between.  Returns (frequencies, what cosines and sines are multiplied by)."""
    def pair_that_turns(n):
        return dims * math.log(original / (2.0 * math.pi * n)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_that_turns(fast)), 0)
    hi = min(math.ceil(pair_that_turns(slow)), dims - 1)
    f = frequencies(base, dims)
    out = torch.empty_like(f)
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / factor * ramp + f[i] * (1.0 - ramp)
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, pos, freq, interleaved, amplitude=1.0):
    """x [T, heads, D]; len(freq) pairs at the front of a head turn by pos * freq: (2i, 2i + 1), or (i, i + len(freq)); the
    rest pass."""
    n = len(freq)
    y = x.clone()
    for i in range(n):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + n)
        ang = pos.to(F64) * freq[i]
        c, s = (amplitude * torch.cos(ang))[:, None], (amplitude * torch.sin(ang))[:, None]
        y[..., a] = x[..., a] * c - x[..., b] * s
        y[..., b] = x[..., b] * c + x[..., a] * s
    return y


def causal(T, chunk=None):
    """[T, T] bool: query i sees key j when j <= i and, with chunks, both lie in the same one (counted from 0)."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    see = j <= i
    if chunk is not None:
        see = see & (i // chunk == j // chunk)
    return see


def softmax_weights(s, see):
    return torch.softmax(s.masked_fill(~see, -math.inf), dim=-1)


def sigmoid_weights(s, see, bias):
    return torch.where(see, torch.sigmoid(s + bias), torch.zeros_like(s))


def wkv_memory(r, k, v, w, u):
    """Per head o_t = (S + diag(u) k_t v_t^T)^T r_t, then S <- diag(w_t) S + k_t v_t^T, from S = 0.
    r, k, w [T, H, D], v [T, H, Dv], u [H, D]."""
    T, H, D = r.shape
    out = torch.zeros((T, H, v.shape[-1]), dtype=F64)
    for h in range(H):
        S = torch.zeros((D, v.shape[-1]), dtype=F64)
        for t in range(T):
            kv = torch.outer(k[t, h], v[t, h])
            out[t, h] = (S + u[h][:, None] * kv).t() @ r[t, h]
            S = w[t, h][:, None] * S + kv
    return out


# ----------------------------------------------------------------------------- mixers
def latent_attention(h, W, p, m, eps, rnd=_ident):
    """Queries through a normed latent; per head a key [W_uk c | the shared rotated part] and a value W_uv c from a normed
    latent c; softmax over all earlier keys; the heads' outputs gated number by number."""
    T = h.shape[0]
    H, D, R, Dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    cq = rnd(rms_unit(rnd(lin(W[p + "dq"], h)), eps) * W[p + "dq.norm"].to(F64))
    q = rnd(lin(W[p + "uq"], cq)).view(T, H, D + R)
    down = rnd(lin(W[p + "dkv"], h))
    c = rnd(rms_unit(down[:, :rank], eps) * W[p + "dkv.norm"].to(F64))
    rot = m["rot"]
    if rot.get("scaling") is not None:
        sc = rot["scaling"]
        freq, amp = stretched_frequencies(rot["base"], rot["dims"], sc["factor"], sc["original"], sc["fast"], sc["slow"])
    else:
        freq, amp = frequencies(rot["base"], rot["dims"]), 1.0
    q_rot = rnd(rotate(q[..., D:], pos, freq, True, amp))
    k_rot = rnd(rotate(down[:, None, rank:], pos, freq, True, amp))[:, 0]
    k = lin(W[p + "uk"], c).view(T, H, D)
    v = lin(W[p + "uv"], c).view(T, H, Dv)
    o = torch.zeros((T, H, Dv), dtype=F64)
    for g in range(H):
        s = (q[:, g, :D] @ k[:, g].t() + q_rot[:, g] @ k_rot.t()) * m["scale"]
        o[:, g] = softmax_weights(s, causal(T)) @ v[:, g]
    o = rnd(rnd(o.reshape(T, H * Dv)) * torch.sigmoid(rnd(lin(W[p + "g"], h))))
    return lin(W[p + "o"], o)


def chunked_attention(h, W, p, m, eps, rnd=_ident):
    """Grouped heads; q and k normed over their whole rows, then rotated; unnormalised sigmoid weights within a chunk; the
    heads' outputs gated number by number."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = rms_unit(rnd(lin(W[p + "q"], h)), eps) * W[p + "q.norm"].to(F64)
    k = rms_unit(rnd(lin(W[p + "k"], h)), eps) * W[p + "k.norm"].to(F64)
    v = rnd(lin(W[p + "v"], h)).view(T, G, Dv)
    rot = m.get("rot")
    q, k = q.view(T, H, D), k.view(T, G, D)
    if rot is not None:
        freq = frequencies(rot["base"], rot["dims"])
        q, k = rotate(q, pos, freq, False), rotate(k, pos, freq, False)
    q, k = rnd(q), rnd(k)
    see = causal(T, m["mask"]["size"] if m.get("mask") is not None else None)
    o = torch.zeros((T, H, Dv), dtype=F64)
    for i in range(H):
        g = i // (H // G)
        o[:, i] = sigmoid_weights((q[:, i] @ k[:, g].t()) * m["scale"], see, W[p + "pb"][i].to(F64)) @ v[:, g]
    o = rnd(rnd(o.reshape(T, H * Dv)) * torch.sigmoid(rnd(lin(W[p + "g"], h))))
    return lin(W[p + "o"], o)


def wkv_mixer(h, W, p, m, eps, rnd=_ident):
    """Every projection reads its own mix of the current and the previous token; a matrix memory per head with a decay per
    key channel and token, and a bonus for the current token."""
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    before = torch.cat([torch.zeros((1, h.shape[1]), dtype=F64), h[:-1]], dim=0)

    def mix(n):
        return rnd(h + (before - h) * W[p + "mu." + n].to(F64))

    r, k, v = (rnd(lin(W[p + n], mix(n))).view(T, H, D) for n in ("r", "k", "v"))
    gate = silu(rnd(lin(W[p + "g"], mix("g"))))
    w = torch.exp(-torch.exp(lin(W[p + "w2"], torch.tanh(lin(W[p + "w1"], mix("w")))) + W[p + "w0"].to(F64))).view(T, H, D)
    o = rms_unit(wkv_memory(r, k, v, w, W[p + "u"].to(F64).view(H, D)), eps).reshape(T, H * D)
    return lin(W[p + "o"], rnd(o * W[p + "norm"].to(F64) * gate))


# ----------------------------------------------------------------------------- feed-forward
def squared_relu_expert(h, W, p, rnd=_ident):
    a = torch.clamp(lin(W[p + "up"], h), min=0.0)
    return lin(W[p + "down"], rnd(a * a))


def route(z, top):
    """The ``top`` largest sigmoid scores of each row (ties to the lower index) and those scores."""
    s = torch.sigmoid(z)
    order = torch.sort(s, dim=-1, descending=True, stable=True).indices[:, :top]
    return order, torch.gather(s, 1, order)


def moe_ff(h, W, p, mlp, rnd=_ident):
    """A chosen expert runs on its score times the token's row; the sum of the experts' outputs as they are, plus the shared
    expert times a sigmoid of one number per token."""
    T = h.shape[0]
    top = mlp["router"]["top"]
    ids, wts = route(lin(W[p + "router"], h), top)
    out = torch.zeros((T, W[p + "e0.down"].shape[0]), dtype=F64)
    for t in range(T):
        for c in range(top):
            out[t] += rnd(squared_relu_expert(wts[t, c] * h[t: t + 1], W, f"{p}e{int(ids[t, c])}.", rnd))[0]
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(lin(W[p + "shared.sg"], h)) * rnd(squared_relu_expert(h, W, p + "shared.", rnd))
    return out


# ----------------------------------------------------------------------------- the model
MIXERS = {"latent_attention": latent_attention, "attention": chunked_attention, "wkv": wkv_mixer}


def forward(cfg, W, tokens, rnd=_ident, layers_out=None):
    eps = cfg["norm"]["eps"]
    x = layer_norm(W["embed"].to(F64)[torch.as_tensor(tokens, dtype=torch.long)], W["embed.norm"], eps)
    for i, layer in enumerate(cfg["layers"]):
        h = rnd(plus_short_conv(x, W[f"l{i}.canon1"]))
        branch = rnd(MIXERS[layer["type"]](h, W, f"l{i}.mix.", layer["mixer"], eps, rnd))
        x = x + layer_norm(branch, W[f"l{i}.norm1"], eps) * W[f"l{i}.ls1"].to(F64)
        if layer.get("mlp") is not None:
            branch = rnd(moe_ff(rnd(x), W, f"l{i}.mlp.", layer["mlp"], rnd))
            x = x + layer_norm(branch, W[f"l{i}.norm2"], eps) * W[f"l{i}.ls2"].to(F64)
        if layers_out is not None:
            layers_out.append(x.clone())
    return lin(W["embed"], rnd(layer_norm(x, W["final.norm"], eps)))


def generate_greedy(cfg, W, prompt, steps):
    toks = list(prompt)
    for _ in range(steps):
        toks.append(int(forward(cfg, W, toks)[-1].argmax()))
    return toks[len(prompt):]
