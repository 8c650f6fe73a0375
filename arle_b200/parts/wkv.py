"""RWKV-style time mixing: a recurrent mixer whose projections each read a mix of their own of the current and the previous
token, with a matrix memory per head, a decay per key channel and token, and a bonus for the current token.

With h' the row of the token before (zeros before a request's first), mix_s = h + (h' - h) * mu_s for s in r, k, v, g, w:

    r, k, v = W_r mix_r, W_k mix_k, W_v mix_v  (heads x dim),  gate = silu(W_g mix_g)
    w = exp(-exp(W_w2 tanh(W_w1 mix_w) + w0))                        per head and key channel
    o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t,    S_t = diag(w_t) S_(t-1) + k_t v_t^T

o is divided by its root mean square per head, the heads side by side are multiplied by a weight of all heads' size and by the
gate, and go through the output projection.  The state (S, float32, and the previous token's row) lives in the request's state
slot.  The decay, its logarithm and the recurrence are float32 in both precisions: the sums of the small matrix W_w1 stay float32
and W_w2 is held in float32.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import ClassVar, Optional, Tuple

import torch

from .. import ops
from .base import Mixer, StateNeed, WeightDecl
from .registry import register_part

MIXES = ("r", "k", "v", "g", "w")      # the order of the mixes in the buffer that one kernel writes


@dataclass(frozen=True)
class WkvSpec:
    prefix: str
    hidden_size: int
    num_heads: int
    head_dim: int                   # keys and values
    decay_rank: int                 # rows of W_w1
    norm_eps: float
    names: Optional[Tuple[Tuple[str, str], ...]] = None    # (role, name after the prefix); see DEFAULT_NAMES
    kind: ClassVar[str] = "wkv"


DEFAULT_NAMES = (("r", "r"), ("k", "k"), ("v", "v"), ("g", "g"), ("o", "o"), ("mu", "mu.{}"), ("decay_in", "w1"), ("decay_out", "w2"),
                 ("decay_bias", "w0"), ("bonus", "u"), ("norm", "norm"))


class WkvMixer(Mixer):
    def __init__(self, spec: WkvSpec):
        if min(spec.num_heads, spec.head_dim, spec.decay_rank) <= 0:
            raise ValueError("wkv: heads, head_dim and decay_rank must be positive")
        if spec.head_dim > 512 or spec.decay_rank > 1024:
            raise ValueError(f"wkv: head_dim {spec.head_dim} (at most 512) or decay_rank {spec.decay_rank} (at most 1,024) not supported")
        self.spec = spec
        self.names = dict(DEFAULT_NAMES)
        self.names.update(dict(spec.names or ()))
        self.inner = spec.num_heads * spec.head_dim
        self.memory = spec.num_heads * spec.head_dim * spec.head_dim
        self.shift_at = -(-self.memory // 4) * 4            # the previous token's row stands behind the memories
        self.w_rkvg = self.w_low = self.w_decay = self.w_o = self.mu = self.decay_bias = self.bonus = self.norm = None

    def _name(self, role: str, of: str = "") -> str:
        return self.spec.prefix + self.names[role].format(of)

    # ---------------------------------------------------------------- weights
    def weight_decls(self):
        s, N = self.spec, self.inner
        return (tuple(WeightDecl(self._name("mu", m), (s.hidden_size,), init="around_zero") for m in MIXES)
                + tuple(WeightDecl(self._name(n), (N, s.hidden_size)) for n in ("r", "k", "v", "g"))
                + (WeightDecl(self._name("decay_in"), (s.decay_rank, s.hidden_size)), WeightDecl(self._name("decay_out"), (N, s.decay_rank)),
                   WeightDecl(self._name("decay_bias"), (N,), init="around_zero"),
                   WeightDecl(self._name("bonus"), (s.num_heads, s.head_dim), init="around_zero"), WeightDecl(self._name("norm"), (N,), init="gain"),
                   WeightDecl(self._name("o"), (s.hidden_size, N))))

    def load(self, tensors, dtype, device):
        def kept(ts):
            return dtype if dtype == torch.bfloat16 else (torch.float32 if any(t.dtype == torch.float32 for t in ts) else torch.bfloat16)

        mats = [tensors[self._name(n)] for n in ("r", "k", "v", "g")]
        self.w_rkvg = torch.stack([m.to(device=device, dtype=kept(mats)) for m in mats]).contiguous()
        low, o = tensors[self._name("decay_in")], tensors[self._name("o")]
        self.w_low = low.to(device=device, dtype=kept([low])).contiguous()
        self.w_o = o.to(device=device, dtype=kept([o])).contiguous()
        self.w_decay = tensors[self._name("decay_out")].to(device=device, dtype=torch.float32).t().contiguous()       # [rank, heads * dim]
        self.decay_bias, self.bonus, self.norm = (tensors[self._name(n)].to(device=device, dtype=torch.float32).reshape(-1).contiguous()
                                                  for n in ("decay_bias", "bonus", "norm"))
        self.mu = torch.stack([tensors[self._name("mu", m)].to(device=device, dtype=torch.float32) for m in MIXES]).contiguous()

    def weight_bytes(self):
        return sum(t.numel() * t.element_size() for t in (self.w_rkvg, self.w_low, self.w_decay, self.w_o))

    def scratch_elements_per_token(self):
        # the mixes, the four projections and the gated output in the activation type; decay and read-out in float32
        return (len(MIXES) + 1) * self.spec.hidden_size + 9 * self.inner + 2 * self.spec.decay_rank

    # ------------------------------------------------------------------ state
    def state_need(self):
        return StateNeed((self.shift_at + -(-self.spec.hidden_size // 4) * 4,), torch.float32)

    def can_sink(self, num_rows):
        return ops.fused_gemm_shape_ok(num_rows, self.w_o)

    # ---------------------------------------------------------------- forward
    def forward(self, x, ctx, cache, state, sink=None):
        s = self.spec
        T = x.shape[0]
        H, D, N = s.num_heads, s.head_dim, self.inner
        mixes = ctx.ws.get("wkv_mixes", (len(MIXES), T, s.hidden_size), x.dtype)
        ops.token_shift(x, self.mu, state[:, self.shift_at: self.shift_at + s.hidden_size], ctx.q_indptr, ctx.row_of_token, ctx.state_slots, mixes,
                        ctx.max_q_len)
        proj = ctx.ws.get("wkv_in", (4, T, N), x.dtype)
        for i in range(4):
            ops.gemm(mixes[i], self.w_rkvg[i], proj[i])
        low = ctx.ws.get("wkv_low", (T, s.decay_rank), torch.float32)
        ops.gemm(mixes[4], self.w_low, low)
        decay = ctx.ws.get("wkv_decay", (T, N), torch.float32)
        ops.gla_decay(low, self.w_decay, self.decay_bias, 1.0, decay, form="double_exp")
        o = ctx.ws.get("wkv_o", (T, N), torch.float32)
        ops.gla_scan(proj[0], proj[1], proj[2], decay, state, ctx.q_indptr, ctx.state_slots, o, H, D, D, 1.0, ctx.max_q_len, bonus=self.bonus)
        gated = ctx.ws.get("wkv_gated", (T, N), x.dtype)
        ops.gla_out(o, proj[3], self.norm, s.norm_eps, 1.0, gated, H, D)
        out = ctx.ws.get("mixer_out", (T, s.hidden_size), x.dtype)
        return None if ops.gemm(gated, self.w_o, out, sink=sink) else out


register_part(WkvSpec.kind, WkvMixer)
