"""Pre-norm block: x <- x + mixer(norm(x)); x <- x + ffn(norm(x)) (the second half is absent when the spec names no
feed-forward)
(infer/src/model/qwen3/prefill.rs:618-776).  The block never touches the residual
itself: it hands branch outputs to the ``ResidualStream``, which folds each into
the 32-bit residual inside the kernel of the next norm, the fusion cklxx/arle's
decode path uses (infer/src/model/qwen3/batch_decode.rs:2422-2452)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import ClassVar

import torch

from .base import Block, StateNeed, WeightDecl
from .registry import build_part, register_part


@dataclass(frozen=True)
class PreNormBlockSpec:
    mixer_norm: object
    mixer: object
    ffn_norm: object = None         # None together with ffn: the block is its mixer half alone
    ffn: object = None
    kind: ClassVar[str] = "prenorm_block"


class PreNormBlock(Block):
    def __init__(self, spec: PreNormBlockSpec):
        self.spec = spec
        self.mixer_norm = build_part(spec.mixer_norm)
        self.mixer = build_part(spec.mixer)
        if (spec.ffn is None) != (spec.ffn_norm is None):
            raise ValueError("a pre-norm block has a feed-forward and its norm, or neither")
        self.ffn_norm = build_part(spec.ffn_norm) if spec.ffn_norm is not None else None
        self.ffn = build_part(spec.ffn) if spec.ffn is not None else None
        self._parts = tuple(p for p in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn) if p is not None)

    def weight_decls(self):
        return tuple(d for p in self._parts for d in p.weight_decls())

    def load(self, tensors, dtype, device):
        for p in self._parts:
            p.load(tensors, dtype, device)

    def weight_bytes(self):
        return sum(p.weight_bytes() for p in self._parts)

    def scratch_elements_per_token(self):
        # the two normalised inputs and the larger of the two branches' buffers
        if self.ffn is None:
            return self.mixer_norm.scratch_elements_per_token() + self.mixer.scratch_elements_per_token()
        return (self.mixer_norm.scratch_elements_per_token() + self.ffn_norm.scratch_elements_per_token()
                + max(self.mixer.scratch_elements_per_token(), self.ffn.scratch_elements_per_token()))

    def entry(self):
        return self.mixer_norm, self.mixer

    def forward(self, stream, ctx, cache, state):
        T = ctx.num_tokens
        h = stream.normed(self.mixer_norm, "normed_a")
        if self.ffn is None:
            nxt = stream.next_entry
            sink = stream.sink_for(nxt[0], nxt[1], "normed_a", last=True) if nxt is not None and self.mixer.can_sink(T) else None
            stream.add(self.mixer.forward(h, ctx, cache, state, sink=sink) if sink is not None else self.mixer.forward(h, ctx, cache, state))
            return
        # where a branch's last product can add into the residual and leave the next norm's input behind,
        # and that norm's reader can apply the norm's factor itself, the norm between them is no kernel
        sink = stream.sink_for(self.ffn_norm, self.ffn, "normed_b") if self.mixer.can_sink(T) else None
        if sink is not None:
            stream.add(self.mixer.forward(h, ctx, cache, state, sink=sink))
        else:
            stream.add(self.mixer.forward(h, ctx, cache, state))
        h = stream.normed(self.ffn_norm, "normed_b")
        nxt = stream.next_entry
        sink = stream.sink_for(nxt[0], nxt[1], "normed_a", last=True) if nxt is not None and self.ffn.can_sink(T) else None
        if sink is not None:
            stream.add(self.ffn.forward(h, ctx, sink=sink))
        else:
            stream.add(self.ffn.forward(h, ctx))


register_part(PreNormBlockSpec.kind, PreNormBlock)


@dataclass(frozen=True)
class OutputNormBlockSpec:
    """x <- x + norm(mixer(x)); x <- x + norm(ffn(x)): the norms stand on the sublayers' outputs, the sublayers read the
    residual as it is (the second half is absent when the spec names no feed-forward).  With ``conv_taps`` the mixer reads
    x + conv(x) instead, a causal convolution over time on every channel (stored weight ``conv_name`` [size, taps], no bias,
    zeros before a sequence's start)."""
    mixer_norm: object
    mixer: object
    ffn_norm: object = None
    ffn: object = None
    conv_taps: int = 0              # 0: no convolution
    conv_name: str = ""
    conv_size: int = 0              # the model width, with a convolution
    kind: ClassVar[str] = "outnorm_block"


class OutputNormBlock(Block):
    """The norm needs ``add_normed(resid, branch, copy)`` (``RmsNorm`` has it): the branch's norm, the sum into the 32-bit
    residual and the rounded copy that the next sublayer reads are one kernel.

    The input convolution reads the 32-bit residual itself.  Its memory, a request's last taps - 1 residual rows in float32,
    stands in front of the mixer's state in one row per request slot (a mixer behind a convolution keeps a flat float32
    state).  In a step of decoded tokens only it runs inside the kernel that ends the block before."""

    scales_branches = False

    def __init__(self, spec: OutputNormBlockSpec):
        self.spec = spec
        self.mixer_norm = build_part(spec.mixer_norm)
        self.mixer = build_part(spec.mixer)
        if (spec.ffn is None) != (spec.ffn_norm is None):
            raise ValueError("a block has a feed-forward and its norm, or neither")
        self.ffn_norm = build_part(spec.ffn_norm) if spec.ffn_norm is not None else None
        self.ffn = build_part(spec.ffn) if spec.ffn is not None else None
        self._parts = tuple(p for p in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn) if p is not None)
        for n in (self.mixer_norm, self.ffn_norm):
            if n is not None and not hasattr(n, "add_normed"):
                raise ValueError(f"norm {type(n).__name__} cannot stand on a branch's output (no add_normed)")
        if spec.conv_taps < 0 or (spec.conv_taps and (spec.conv_size <= 0 or not spec.conv_name)):
            raise ValueError("a block's input convolution needs taps, a size and its weight's name")
        self.conv = None
        n = spec.conv_size * (spec.conv_taps - 1) if spec.conv_taps else 0
        self.conv_state = -(-n // 4) * 4                # columns of the state row that belong to the convolution
        self._mixer_state = self.mixer.state_need()
        if spec.conv_taps and self._mixer_state is not None and (self._mixer_state.dtype != torch.float32 or len(self._mixer_state.shape) != 1):
            raise ValueError("a mixer behind an input convolution needs a flat float32 state")

    def weight_decls(self):
        s = self.spec
        own = (WeightDecl(s.conv_name, (s.conv_size, s.conv_taps), init="around_zero"),) if s.conv_taps else ()
        return tuple(d for p in self._parts for d in p.weight_decls()) + own

    def load(self, tensors, dtype, device):
        for p in self._parts:
            p.load(tensors, dtype, device)
        if self.spec.conv_taps:
            w = tensors[self.spec.conv_name].to(device=device, dtype=torch.float32).t().contiguous().clone()        # [taps, size]
            w[-1] += 1.0                                # x + conv(x) as one sum
            self.conv = w

    def state_need(self):
        if not self.conv_state:
            return self._mixer_state
        return StateNeed((self.conv_state + (self._mixer_state.shape[0] if self._mixer_state is not None else 0),), torch.float32)

    def input_conv(self, state):
        if self.conv is None:
            return None
        return self.conv, (state[:, : self.spec.conv_size * (self.spec.conv_taps - 1)] if self.conv_state else None)

    def weight_bytes(self):
        return sum(p.weight_bytes() for p in self._parts)

    def scratch_elements_per_token(self):
        width = self.mixer_norm.scratch_elements_per_token()
        return 2 * width + max(self.mixer.scratch_elements_per_token(), self.ffn.scratch_elements_per_token() if self.ffn is not None else 0)

    def forward(self, stream, ctx, cache, state):
        conv = self.input_conv(state)
        h = stream.plain("plain_a") if conv is None else stream.convolved(conv, ctx, "convolved")
        if self.conv_state:
            state = state[:, self.conv_state:] if self._mixer_state is not None else None
        branch = self.mixer.forward(h, ctx, cache, state)
        # what the next block reads: the residual's convolution (then no rounded copy of the residual is wanted), or its copy
        leaves = None if stream.next_conv is not None else "plain_a"
        if self.ffn is None:
            if not stream.add_normed_then_conv(self.mixer_norm, branch, ctx, "convolved"):
                stream.add_normed(self.mixer_norm, branch, leaves)
            return
        stream.add_normed(self.mixer_norm, branch, "plain_b")
        h = stream.plain("plain_b")
        branch = self.ffn.forward(h, ctx)
        if not stream.add_normed_then_conv(self.ffn_norm, branch, ctx, "convolved"):
            stream.add_normed(self.ffn_norm, branch, leaves)


register_part(OutputNormBlockSpec.kind, OutputNormBlock)


@dataclass(frozen=True)
class SandwichBlockSpec:
    """x <- x + post(mixer(pre(x))); x <- x + post'(ffn(pre'(x))): a norm on every sublayer's input AND on its output (the
    second half is absent when the spec names no feed-forward)."""
    mixer_norm: object
    mixer: object
    mixer_post_norm: object
    ffn_norm: object = None
    ffn: object = None
    ffn_post_norm: object = None
    kind: ClassVar[str] = "sandwich_block"


class SandwichBlock(Block):
    """A sublayer's output norm, the sum into the 32-bit residual and the next sublayer's input norm are one kernel
    (``ResidualStream.add_normed_before_norm``): the stream keeps the branch until the next ``normed(...)``."""

    scales_branches = False

    def __init__(self, spec: SandwichBlockSpec):
        self.spec = spec
        given = [spec.ffn is not None, spec.ffn_norm is not None, spec.ffn_post_norm is not None]
        if any(given) != all(given):
            raise ValueError("a block has a feed-forward with both of its norms, or none of the three")
        self.mixer_norm = build_part(spec.mixer_norm)
        self.mixer = build_part(spec.mixer)
        self.mixer_post_norm = build_part(spec.mixer_post_norm)
        self.ffn_norm = build_part(spec.ffn_norm) if spec.ffn is not None else None
        self.ffn = build_part(spec.ffn) if spec.ffn is not None else None
        self.ffn_post_norm = build_part(spec.ffn_post_norm) if spec.ffn is not None else None
        self._parts = tuple(p for p in (self.mixer_norm, self.mixer, self.mixer_post_norm, self.ffn_norm, self.ffn, self.ffn_post_norm)
                            if p is not None)
        for n in (self.mixer_post_norm, self.ffn_post_norm):
            if n is not None and not hasattr(n, "add_normed"):
                raise ValueError(f"norm {type(n).__name__} cannot stand on a branch's output (no add_normed)")

    def weight_decls(self):
        return tuple(d for p in self._parts for d in p.weight_decls())

    def load(self, tensors, dtype, device):
        for p in self._parts:
            p.load(tensors, dtype, device)

    def weight_bytes(self):
        return sum(p.weight_bytes() for p in self._parts)

    def scratch_elements_per_token(self):
        width = self.mixer_norm.scratch_elements_per_token()
        return 2 * width + max(self.mixer.scratch_elements_per_token(), self.ffn.scratch_elements_per_token() if self.ffn is not None else 0)

    def forward(self, stream, ctx, cache, state):
        h = stream.normed(self.mixer_norm, "normed_a")
        stream.add_normed_before_norm(self.mixer_post_norm, self.mixer.forward(h, ctx, cache, state))
        if self.ffn is not None:
            h = stream.normed(self.ffn_norm, "normed_b")
            stream.add_normed_before_norm(self.ffn_post_norm, self.ffn.forward(h, ctx))


register_part(SandwichBlockSpec.kind, SandwichBlock)
