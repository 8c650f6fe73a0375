"""Gated feed-forward: down(act(gate(x)) * up(x)), no biases; act is silu (SwiGLU,
infer/src/model/qwen3/prefill.rs:291-337) or the tanh form of gelu.  Gate and up are packed into one [2I, H]
matrix at load (cklxx/arle offers a packed layout as an option,
infer/src/model/qwen3/weights.rs:98-122); here row 2i is gate_i and row 2i + 1 is up_i, so
that the kernel that forms both sums of a pair can apply the gate itself."""
from __future__ import annotations

from dataclasses import dataclass
from typing import ClassVar, Tuple

import torch

from .. import ops
from .base import FeedForward, WeightDecl
from .registry import register_part


@dataclass(frozen=True)
class GatedMlpSpec:
    prefix: str
    hidden_size: int
    intermediate_size: int
    activation: str = "silu"        # "silu", "gelu_tanh" or "clamped_glu"
    names: Tuple[str, str, str] = ("gate_proj.weight", "up_proj.weight", "down_proj.weight")   # after the prefix
    act_limit: float = 0.0          # "clamped_glu": g = min(gate x, limit), u = clamp(up x, +-limit), g sigmoid(act_alpha g) (u + 1)
    act_alpha: float = 1.702
    kind: ClassVar[str] = "gated_mlp"


class GatedMlp(FeedForward):
    def __init__(self, spec: GatedMlpSpec):
        self.clamped = spec.activation == "clamped_glu"
        if self.clamped and not spec.act_limit > 0:
            raise ValueError("gated feed-forward: the clamped activation needs a positive act_limit")
        if spec.activation not in ops.ACTIVATIONS and not self.clamped:
            raise ValueError(f"activation {spec.activation!r} not supported by the gated feed-forward "
                             f"({', '.join(ops.ACTIVATIONS)})")
        self.spec = spec
        self.w_gate_up = self.w_down = None

    def weight_decls(self):
        s, p = self.spec, self.spec.prefix
        g, u, d = s.names
        return (WeightDecl(p + g, (s.intermediate_size, s.hidden_size)),
                WeightDecl(p + u, (s.intermediate_size, s.hidden_size)),
                WeightDecl(p + d, (s.hidden_size, s.intermediate_size)))

    def load(self, tensors, dtype, device):
        p = self.spec.prefix
        g, u, d = (tensors[p + n] for n in self.spec.names)
        wt = dtype if dtype == torch.bfloat16 else (torch.float32 if torch.float32 in (g.dtype, u.dtype) else torch.bfloat16)
        g, u = g.to(device=device, dtype=wt), u.to(device=device, dtype=wt)
        self.w_gate_up = torch.stack([g, u], dim=1).reshape(2 * g.shape[0], g.shape[1]).contiguous()
        self.w_down = d.to(device=device, dtype=dtype if dtype == torch.bfloat16 else d.dtype).contiguous()

    def weight_bytes(self):
        return sum(t.numel() * t.element_size() for t in (self.w_gate_up, self.w_down))

    def scratch_elements_per_token(self):
        return 3 * self.spec.intermediate_size + self.spec.hidden_size

    def takes_scaled_rows(self, num_rows):
        return not self.clamped and ops.fused_gemm_shape_ok(num_rows, self.w_gate_up, gated=True)

    def can_sink(self, num_rows):
        return ops.fused_gemm_shape_ok(num_rows, self.w_down)

    # the feed-forward up to its last product
    def pre_output_width(self):
        return None if self.clamped else self.spec.intermediate_size

    def output_weight(self):
        return self.w_down

    def forward_pre(self, x, ctx, into):
        s = self.spec
        gu = ctx.ws.get("gate_up", (x.shape[0], 2 * s.intermediate_size), x.dtype)
        ops.gemm_act_mul(x, self.w_gate_up, gu, into, s.activation)

    def forward(self, x, ctx, sink=None):
        s = self.spec
        T = x.shape[0]
        gu = ctx.ws.get("gate_up", (T, 2 * s.intermediate_size), x.dtype)
        act = ctx.ws.get("ffn_act", (T, s.intermediate_size), x.dtype)
        if self.clamped:
            ops.gemm(x, self.w_gate_up, gu)
            ops.clamped_glu(gu, act, s.act_limit, s.act_alpha)
        else:
            ops.gemm_act_mul(x, self.w_gate_up, gu, act, s.activation)
        out = ctx.ws.get("ffn_out", (T, s.hidden_size), x.dtype)
        if ops.gemm(act, self.w_down, out, sink=sink):
            return None                       # summed into the residual by the product itself
        return out


register_part(GatedMlpSpec.kind, GatedMlp)


@dataclass(frozen=True)
class UngatedMlpSpec:
    """down(act(up(x))), no biases; ``activation`` "square_relu": max(z, 0)^2."""
    prefix: str
    hidden_size: int
    intermediate_size: int
    activation: str = "square_relu"
    names: Tuple[str, str] = ("up_proj.weight", "down_proj.weight")     # after the prefix
    kind: ClassVar[str] = "ungated_mlp"


class UngatedMlp(FeedForward):
    def __init__(self, spec: UngatedMlpSpec):
        if spec.activation != "square_relu":
            raise ValueError(f"activation {spec.activation!r} not supported by the ungated feed-forward (square_relu)")
        self.spec = spec
        self.w_up = self.w_down = None

    def weight_decls(self):
        s = self.spec
        return (WeightDecl(s.prefix + s.names[0], (s.intermediate_size, s.hidden_size)),
                WeightDecl(s.prefix + s.names[1], (s.hidden_size, s.intermediate_size)))

    def load(self, tensors, dtype, device):
        up, down = (tensors[self.spec.prefix + n] for n in self.spec.names)
        self.w_up, self.w_down = (t.to(device=device, dtype=dtype if dtype == torch.bfloat16 else t.dtype).contiguous() for t in (up, down))

    def weight_bytes(self):
        return sum(t.numel() * t.element_size() for t in (self.w_up, self.w_down))

    def scratch_elements_per_token(self):
        return self.spec.intermediate_size + self.spec.hidden_size

    def takes_scaled_rows(self, num_rows):
        return ops.fused_gemm_shape_ok(num_rows, self.w_up)

    def can_sink(self, num_rows):
        return ops.fused_gemm_shape_ok(num_rows, self.w_down)

    def forward(self, x, ctx, sink=None):
        s = self.spec
        T = x.shape[0]
        act = ctx.ws.get("ffn_act", (T, s.intermediate_size), x.dtype)
        ops.gemm_square_relu(x, self.w_up, act)
        out = ctx.ws.get("ffn_out", (T, s.hidden_size), x.dtype)
        return None if ops.gemm(act, self.w_down, out, sink=sink) else out


register_part(UngatedMlpSpec.kind, UngatedMlp)
