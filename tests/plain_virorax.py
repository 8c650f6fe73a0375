"""A plain, slow implementation of the Virorax design: float64 torch on the CPU, whole sequences,
no cache, no batching, one function per mechanism.  It shares no code with the package's model
path; the tests compare the engine with it.

A model is (config dict in the form of config.json, {tensor name: tensor}).  ``forward`` returns
the logits of every position and, on request, the residual after every layer run.  ``rnd`` is applied
to every stored activation (identity by default; rounding to bfloat16 gives the tests the size of
what rounding alone does).

A layer norms before each sublayer and scales what the sublayer returns: x <- x + m mixer(n1(x)),
x <- x + m ff(n2(x)).  Notation: h is a sublayer's input [T, width]; positions count from 0.
"""
from __future__ import annotations

import torch

F64 = torch.float64


def _ident(x):
    return x


def round_bf16(x):
    return x.to(torch.float32).to(torch.bfloat16).to(F64)


def lin(W, x, b=None):
    """Rows of x through a matrix stored [out, in], plus a bias."""
    y = x @ W.to(F64).t()
    return y if b is None else y + b.to(F64)


# ----------------------------------------------------------------------------- small functions
def unit_rms(x, eps):
    """Each last axis divided by its root mean square, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w.to(F64)


def silu(z):
    return z * torch.sigmoid(z)


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def rotate_halves(x, pos, base, dims):
    """x [T, heads, D]; of the first ``dims`` numbers of a head, number i turns with number i + dims/2 by
    the angle pos * base^(-2i/dims); the rest pass."""
    if not dims:
        return x
    half = dims // 2
    freq = torch.pow(torch.tensor(float(base), dtype=F64), -2.0 * torch.arange(half, dtype=F64) / dims)
    ang = (pos.to(F64)[:, None] * freq[None, :])[:, None, :]
    c, s = torch.cos(ang), torch.sin(ang)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def within_window(T, window=None):
    """[T, T] bool: query i sees key j when 0 <= i - j (< window)."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) if window is None else (d >= 0) & (d < window)


def sink_attention(q, k, v, scale, see, sinks):
    """q [T, H, D], k [T, G, D], v [T, G, Dv], sinks [H] (or None); query head h reads key head h // (H / G).  A key's weight
    is e^s_j / (e^sink_h + sum over visible keys of e^s).  Returns [T, H, Dv]."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros((T, H, v.shape[-1]), dtype=F64)
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].t()) * scale
        s = s.masked_fill(~see, float("-inf"))
        if sinks is None:
            out[:, h] = torch.softmax(s, dim=-1) @ v[:, h // per]
        else:
            with_sink = torch.cat([s, sinks[h].to(F64).expand(T, 1)], dim=-1)
            out[:, h] = torch.softmax(with_sink, dim=-1)[:, :-1] @ v[:, h // per]
    return out


def decaying_memory(q, k, v, decay):
    """Per head S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, from S = 0.  q, k [T, H, D], v [T, H, Dv]."""
    T, H, D = q.shape
    out = torch.zeros((T, H, v.shape[-1]), dtype=F64)
    for h in range(H):
        S = torch.zeros((D, v.shape[-1]), dtype=F64)
        for t in range(T):
            S = float(decay[h]) * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.t() @ q[t, h]
    return out


# ----------------------------------------------------------------------------- mixers
def attention_mixer(h, W, p, m, eps, rnd=_ident):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q, k, v = (rnd(lin(W[p + n], h, W[p + n + ".b"])) for n in ("q", "k", "v"))
    q, k, v = q.view(T, H, D), k.view(T, G, D), v.view(T, G, Dv)
    q, k = rms_norm(q, W[p + "q.norm"], eps), rms_norm(k, W[p + "k.norm"], eps)
    if m.get("rot") is not None:
        q, k = (rotate_halves(t, pos, m["rot"]["base"], m["rot"]["dims"]) for t in (q, k))
    q, k = rnd(q), rnd(k)
    see = within_window(T, m["mask"]["size"] if m.get("mask") is not None else None)
    o = rnd(sink_attention(q, k, v, m["scale"], see, W[p + "sink"]))
    gate = torch.sigmoid(rnd(lin(W[p + "g"], h)))                # one number per head
    o = rnd(o * gate[:, :, None])
    return lin(W[p + "o"], o.reshape(T, H * Dv))


def retention_mixer(h, W, p, m, eps, rnd=_ident):
    T = h.shape[0]
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q, k, v = (rnd(lin(W[p + n], h)) for n in ("q", "k", "v"))
    q, k, v = q.view(T, H, D), k.view(T, H, D), v.view(T, H, Dv)
    if m.get("rot") is not None:
        q, k = (rotate_halves(t, pos, m["rot"]["base"], m["rot"]["dims"]) for t in (q, k))
    o = decaying_memory(q, k * float(D) ** -0.5, v, m["decay"])
    o = unit_rms(o, eps).reshape(T, H * Dv)
    o = rnd(o * silu(rnd(lin(W[p + "g"], h))))
    return lin(W[p + "o"], o)


# ----------------------------------------------------------------------------- feed-forward
def square_relu_ff(h, W, p, rnd=_ident):
    return lin(W[p + "down"], rnd(torch.clamp(lin(W[p + "up"], h), min=0.0) ** 2))


# ----------------------------------------------------------------------------- the model
def runs(cfg):
    """The layer runs in order: (layer, starts a pass after the first of a loop)."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if loop is None:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    out = [(i, False) for i in range(a)]
    for t in range(times):
        out += [(i, t > 0 and i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n)]


def forward(cfg, W, tokens, rnd=_ident, layers_out=None):
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"].to(F64)[ids] + W["pos"].to(F64)[: len(ids)]
    start = x
    for i, again in runs(cfg):
        layer = cfg["layers"][i]
        p, m = f"l{i}.mix.", layer["mixer"]
        if again:
            x = x + start
        h = rnd(rms_norm(x, W[f"l{i}.norm1"], eps))
        if layer["type"] == "attention":
            branch = attention_mixer(h, W, p, m, eps, rnd)
        elif layer["type"] == "retention":
            branch = retention_mixer(h, W, p, m, eps, rnd)
        else:
            raise ValueError(layer["type"])
        x = x + mult * rnd(branch)
        if layer.get("mlp") is not None:
            h = rnd(rms_norm(x, W[f"l{i}.norm2"], eps))
            x = x + mult * rnd(square_relu_ff(h, W, f"l{i}.mlp.", rnd))
        if layers_out is not None:
            layers_out.append(x.clone())
    logits = lin(W["embed"], rnd(rms_norm(x, W["final.norm"], eps)))
    return capped(logits, cfg["logit_softcap"]) if cfg.get("logit_softcap") else logits


def generate_greedy(cfg, W, prompt, steps):
    toks = list(prompt)
    for _ in range(steps):
        toks.append(int(forward(cfg, W, toks)[-1].argmax()))
    return toks[len(prompt):]
