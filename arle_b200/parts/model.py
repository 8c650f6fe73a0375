"""A decoder model put together from a ``ModelSpec``: embedding table, blocks,
the schedule that orders them, final norm and output projection.

``DecoderModel.forward(ctx)`` runs exactly the tokens of one step (``ctx`` is a
``StepContext``) and returns float32 logits at the wanted rows.  It is the only
forward pass of the package: generation, the trace replayer and the benchmark
all go through it.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence

import torch

from .. import ops
from ..config.model_spec import ModelSpec
from .base import WeightDecl
from .registry import build_part, register_model


class ResidualStream:
    """The 32-bit residual of a step and the branch output not yet summed into it.

    ``add(delta)`` only remembers the branch output; the next ``normed(...)`` sums
    it into the residual and normalises in one kernel.  Two ``add`` calls in a row
    (a block with parallel branches) are summed right away.

    For steps of few rows the norm kernel can disappear altogether: ``sink_for(norm, ...)``
    hands out an ``ops.ResidualSink`` that a branch's last product fills (residual sum, the norm's
    gain, sums of squares), and the ``normed(...)`` of that norm then returns ``ops.ScaledRows``, whose
    per-row factor the next product applies.  ``next_entry`` is what runs after the current block
    (its first norm and that norm's reader), set by the model.

    ``scale`` multiplies every branch output on its way into the residual.  ``start_run(extra)`` (called by the model before
    each run of a block) makes rows of their own join the residual with the branch that is still pending: inside the run's first
    norm, or inside the sink that the run before has filled for it."""

    def __init__(self, resid: torch.Tensor, ws, act_dtype: torch.dtype, scale: float = 1.0):
        self.resid = resid
        self.ws = ws
        self.act_dtype = act_dtype
        self.scale = scale
        self.pending: Optional[torch.Tensor] = None
        self.next_entry = None
        self.next_extra: Optional[torch.Tensor] = None  # what joins the residual right before the next run, set by the model
        self._extra: Optional[torch.Tensor] = None      # what joins it before the run that starts now, not yet summed
        self._sink = None
        self._sinks_made = 0
        self._copy: Optional[torch.Tensor] = None       # the residual as it stands, in the activation type (or None)
        self._normed_branch = None                      # (norm, branch): resid += norm(branch) still to be done
        self.next_conv = None                           # the next block's input convolution and its memory (or None), set by the model
        self._convolved = None                          # (weight, output): already done by the kernel of the sum before it

    def start_run(self, extra: Optional[torch.Tensor]) -> None:
        if extra is None:
            return
        if self._sink is not None and self._sink[1].filled:
            if self._sink[1].extra is not extra:
                raise RuntimeError("a residual sink was filled without the rows that join the residual before this run")
            return
        self._extra = extra
        self._copy = None

    def _sum_pending(self) -> None:
        ops.residual_add(self.resid, self.pending, self.scale)
        self.pending = None

    def _settle(self) -> None:
        """Whatever ``add_normed_before_norm`` or ``start_run`` left to the next norm is summed into the residual now."""
        if self._extra is not None:
            ops.residual_add(self.resid, self._extra)
            self._extra = None
        if self._normed_branch is not None:
            norm, branch = self._normed_branch
            self._normed_branch = None
            norm.add_normed(self.resid, branch, None)
            self._copy = None

    def add_normed_before_norm(self, norm, branch: torch.Tensor) -> None:
        """resid += norm(branch) for a block whose next sublayer norms its input again: the sum waits for that
        ``normed(...)``, which does both norms in one kernel when it can (``Norm.apply_after``)."""
        self._settle()
        if self.pending is not None:
            self._sum_pending()
        self._normed_branch = (norm, branch)
        self._copy = None

    def add(self, delta: Optional[torch.Tensor]) -> None:
        """``delta`` None: the branch has already put its output into the residual (through a sink)."""
        if delta is None:
            return
        self._settle()
        if self.pending is not None:
            self._sum_pending()
        self.pending = delta
        self._copy = None

    # Blocks whose norms stand on the branches' outputs: the sublayers read the residual as it is.
    def plain(self, buffer_name: str) -> torch.Tensor:
        """The residual as a sublayer's input: itself in float32, its rounding to the activation type otherwise
        (written by the ``add_normed`` before it, or by a pass of its own at the model's first block)."""
        self._settle()
        if self.pending is not None:
            self._sum_pending()
            self._copy = None
        if self.act_dtype == torch.float32:
            return self.resid
        if self._copy is None:
            self._copy = self.ws.get(buffer_name, tuple(self.resid.shape), self.act_dtype)
            ops.branch_norm_add(self.resid, None, None, 0.0, self._copy)
        return self._copy

    def convolved(self, conv, ctx, buffer_name: str) -> torch.Tensor:
        """The causal convolution of the residual over time that a block puts before its mixer; ``conv`` is what the block's
        ``input_conv`` returned."""
        weight, memory = conv
        if self._convolved is not None:
            done_for, out = self._convolved
            self._convolved = None
            if done_for is not weight:
                raise RuntimeError("an input convolution was run for another block than the one that runs next")
            return out
        self._settle()
        if self.pending is not None:
            self._sum_pending()
            self._copy = None
        out = self.ws.get(buffer_name, tuple(self.resid.shape), self.act_dtype)
        ops.input_conv(self.resid, weight, memory, ctx.q_indptr, ctx.row_of_token, ctx.state_slots, out, ctx.max_q_len)
        return out

    def add_normed_then_conv(self, norm, branch: torch.Tensor, ctx, buffer_name: str) -> bool:
        """resid += norm(branch) as a block's last act, with the next block's input convolution in the same kernel where that
        can be (every row of the step one token, a norm that knows how).  False: nothing was done."""
        if self.next_conv is None or ctx.max_q_len != 1 or not hasattr(norm, "add_normed_conv"):
            return False
        self._settle()
        if self.pending is not None:
            self._sum_pending()
        weight, memory = self.next_conv
        out = self.ws.get(buffer_name, tuple(self.resid.shape), self.act_dtype)
        norm.add_normed_conv(self.resid, branch, weight, memory, ctx.state_slots, out)
        self._copy = None
        self._convolved = (weight, out)
        return True

    def add_normed(self, norm, branch: torch.Tensor, buffer_name: Optional[str]) -> None:
        """resid += norm(branch), and the rounded residual for whoever reads it next (no buffer name: nobody does), in one
        kernel."""
        self._settle()
        if self.pending is not None:
            self._sum_pending()
        copy = None if self.act_dtype == torch.float32 or buffer_name is None else self.ws.get(buffer_name, tuple(self.resid.shape), self.act_dtype)
        norm.add_normed(self.resid, branch, copy)
        self._copy = copy

    def sink_for(self, norm, reader, buffer_name: str, last: bool = False):
        """A sink for the branch that runs now, if the norm that follows it can be deferred and its
        reader takes rows without their factor; else None.  ``last``: the branch is its block's last one (the norm is
        the next run's)."""
        T = self.resid.shape[0]
        self._settle()
        if (norm is None or reader is None or self.pending is not None or self.act_dtype != torch.bfloat16
                or not self.resid.is_cuda or ops.kernel_set() != "fast" or not reader.takes_scaled_rows(T)):
            return None
        d = norm.deferred()
        if d is None:
            return None
        gain, eps = d
        xs = self.ws.get(buffer_name, tuple(self.resid.shape), self.act_dtype)
        # two tables in turn: the one being filled is never the one the running product reads
        ss = self.ws.get(f"row_ss_{self._sinks_made & 1}", ops.SS_TABLE_SHAPE, torch.float32)
        self._sinks_made += 1
        self._sink = (norm, ops.ResidualSink(self.resid, gain, eps, xs, ss, self.scale, self.next_extra if last else None))
        return self._sink[1]

    def normed(self, norm, buffer_name: str):
        if self._sink is not None:
            for_norm, sink = self._sink
            self._sink = None
            if sink.filled:
                if for_norm is not norm or self.pending is not None:
                    raise RuntimeError("a residual sink was filled for another norm than the one that runs next")
                return ops.ScaledRows(sink.xs, sink.ss, sink.eps)
        out = self.ws.get(buffer_name, tuple(self.resid.shape), self.act_dtype)
        if self._normed_branch is not None and self.pending is None and self._extra is None and hasattr(norm, "apply_after"):
            post, branch = self._normed_branch
            if norm.apply_after(self.resid, branch, post, out):
                self._normed_branch = None
                self._copy = None
                return out
        extra = None
        if norm.takes_scaled_delta:
            extra, self._extra = self._extra, None
        self._settle()
        if self.scale == 1.0 and extra is None:
            norm.apply(self.resid, self.pending, None, out, write_resid=self.pending is not None)
        elif norm.takes_scaled_delta:
            norm.apply(self.resid, self.pending, None, out, write_resid=self.pending is not None or extra is not None, delta_scale=self.scale,
                       extra=extra)
        else:
            if self.pending is not None:
                self._sum_pending()
            norm.apply(self.resid, None, None, out, write_resid=False)
        if self.pending is not None or extra is not None:
            self._copy = None
        self.pending = None
        return out

    def normed_rows(self, norm, rows: torch.Tensor, buffer_name: str) -> torch.Tensor:
        """Norm of the rows listed only (the residual itself is left as it is)."""
        self._settle()
        out = self.ws.get(buffer_name, (rows.numel(), self.resid.shape[1]), self.act_dtype)
        if self.scale == 1.0:
            norm.apply(self.resid, self.pending, rows, out, write_resid=False)
        elif norm.takes_scaled_delta:
            norm.apply(self.resid, self.pending, rows, out, write_resid=False, delta_scale=self.scale)
        else:
            if self.pending is not None:
                self._sum_pending()
            norm.apply(self.resid, None, rows, out, write_resid=False)
        return out


def declared_weights(spec: ModelSpec) -> List[WeightDecl]:
    """Every tensor a checkpoint of this model must hold."""
    decls = [WeightDecl(spec.embed_name, (spec.vocab_size, spec.hidden_size))]
    if spec.position_name is not None:
        decls.append(WeightDecl(spec.position_name, (spec.max_position, spec.hidden_size)))
    if spec.embed_norm is not None:
        decls.extend(build_part(spec.embed_norm).weight_decls())
    for b in spec.blocks:
        decls.extend(build_part(b).weight_decls())
    decls.extend(build_part(spec.final_norm).weight_decls())
    if spec.head_name is not None:
        decls.append(WeightDecl(spec.head_name, (spec.vocab_size, spec.hidden_size)))
    names = [d.name for d in decls]
    if len(set(names)) != len(names):
        dup = sorted({n for n in names if names.count(n) > 1})
        raise ValueError("tensor names declared twice: " + ", ".join(dup))
    return decls


class DecoderModel:
    def __init__(self, spec: ModelSpec):
        spec.validate()
        self.spec = spec
        self.blocks = [build_part(b) for b in spec.blocks]
        self.final_norm = build_part(spec.final_norm)
        self.embed_norm = build_part(spec.embed_norm) if spec.embed_norm is not None else None
        self.embed = self.head = self.pos_table = None
        if spec.branch_scale != 1.0 and not all(b.scales_branches for b in self.blocks):
            raise ValueError("a factor on the branches goes with blocks that add a branch's output as it is")
        self.readds_embedding = any(e.add_embedding for e in spec.schedule)
        self.dtype = None
        # cache layers: one per schedule entry that keeps keys of its own
        self.cache_needs = []
        self.entry_cache_layer: List[Optional[int]] = []
        self.state_needs = []
        self.entry_state: List[Optional[int]] = []
        for i, e in enumerate(spec.schedule):
            mixer = self.blocks[e.block].mixer
            need = mixer.cache_need()
            if e.keys_of is not None:
                src = spec.schedule[e.keys_of]
                src_need = self.blocks[src.block].mixer.cache_need()
                if need is None or src_need is None or need.arrays() != src_need.arrays():
                    raise ValueError(f"schedule entry {i} cannot read the cache of entry {e.keys_of}: their per-token arrays differ")
                self.entry_cache_layer.append(self.entry_cache_layer[e.keys_of])
            elif need is not None:
                self.entry_cache_layer.append(len(self.cache_needs))
                self.cache_needs.append(need)
            else:
                self.entry_cache_layer.append(None)
            sneed = self.blocks[e.block].state_need()
            if sneed is not None:
                self.entry_state.append(len(self.state_needs))
                self.state_needs.append(sneed)
            else:
                self.entry_state.append(None)

    # ---------------------------------------------------------------- weights
    def weight_decls(self):
        return declared_weights(self.spec)

    def load(self, tensors: Dict[str, torch.Tensor], dtype: torch.dtype, device) -> "DecoderModel":
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"engine dtype must be bfloat16 or float32, got {dtype}")
        device = torch.device(device)
        self.dtype = dtype

        def matrix(t):
            return t.to(device=device, dtype=dtype if dtype == torch.bfloat16 else t.dtype).contiguous()

        self.embed = matrix(tensors[self.spec.embed_name])
        self.head = self.embed if self.spec.head_name is None else matrix(tensors[self.spec.head_name])
        if self.spec.position_name is not None:
            # the embedding kernel reads both tables in one type
            self.pos_table = matrix(tensors[self.spec.position_name])
            if self.pos_table.dtype != self.embed.dtype:
                if self.embed.dtype == torch.float32:
                    self.pos_table = self.pos_table.to(torch.float32)
                else:
                    raise ValueError("a float32 position table needs a float32 embedding table")
        for b in self.blocks:
            b.load(tensors, dtype, device)
        self.final_norm.load(tensors, dtype, device)
        if self.embed_norm is not None:
            self.embed_norm.load(tensors, dtype, device)
        return self

    def weight_bytes_per_step(self) -> int:
        """Bytes of weights a step reads: every scheduled block once and the output
        projection (the embedding gather reads a few rows only)."""
        n = self.head.numel() * self.head.element_size() + self.final_norm.weight_bytes()
        for e in self.spec.schedule:
            n += self.blocks[e.block].weight_bytes()
        return n

    # ---------------------------------------------------------------- forward
    # The forward pass in three steps that a model class of another arrangement may replace
    # one by one: the residual the blocks start from, the scheduled blocks, the logits.
    def embed_tokens(self, ctx) -> torch.Tensor:
        """The float32 residual [T, hidden] of this step's tokens."""
        resid = ctx.ws.get("residual", (ctx.num_tokens, self.spec.hidden_size), torch.float32)
        start = ctx.ws.get("embedding_output", (ctx.num_tokens, self.spec.hidden_size), torch.float32) if self.readds_embedding else None
        ctx.memo["embedding_output"] = start                 # for the runs before which it is added again
        ops.embedding(ctx.token_ids, self.embed, resid, None, getattr(ctx, "last_token", None),
                      getattr(ctx, "slot_of_token", None), scale=self.spec.embed_scale, pos_table=self.pos_table,
                      positions=ctx.positions if self.pos_table is not None else None, out2=start if self.embed_norm is None else None)
        if self.embed_norm is not None:
            self.embed_norm.apply(resid, None, None, resid, write_resid=False)       # in place: the residual starts normed, in float32
            if start is not None:
                start.copy_(resid)
        return resid

    def run_blocks(self, stream: ResidualStream, ctx) -> None:
        order = self.spec.schedule
        start = ctx.memo.get("embedding_output")

        def state_of(i):
            return ctx.state_view(self.entry_state[i]) if self.entry_state[i] is not None else None

        for i, e in enumerate(order):
            after = self.blocks[order[i + 1].block] if i + 1 < len(order) else None
            stream.next_entry = after.entry() if after is not None else None
            stream.next_extra = start if after is not None and order[i + 1].add_embedding else None
            stream.start_run(start if e.add_embedding else None)
            stream.next_conv = after.input_conv(state_of(i + 1)) if after is not None else None
            cl = self.entry_cache_layer[i]
            cache = ctx.cache_view(cl, writable=e.keys_of is None) if cl is not None else None
            st = state_of(i)
            self.blocks[e.block].forward(stream, ctx, cache, st)

    def logits_at_wanted(self, stream: ResidualStream, ctx) -> torch.Tensor:
        final = stream.normed_rows(self.final_norm, ctx.want_rows, "final_normed")
        logits = ctx.ws.get("logits", (ctx.num_wanted, self.spec.vocab_size), torch.float32)
        ops.gemm(final, self.head, logits)
        if self.spec.logit_scale != 1.0:
            ops.weighted_sum(logits, self.spec.logit_scale, logits, 0.0, logits)
        if self.spec.logit_cap:
            ops.logit_cap(logits, self.spec.logit_cap)
        return logits

    def forward(self, ctx) -> Optional[torch.Tensor]:
        stream = ResidualStream(self.embed_tokens(ctx), ctx.ws, self.dtype, self.spec.branch_scale)
        self.run_blocks(stream, ctx)
        if ctx.num_wanted == 0:
            return None
        return self.logits_at_wanted(stream, ctx)

    def scratch_bytes(self, tokens: int, wanted: int) -> int:
        """Bytes of step buffers a step of this many tokens and wanted rows holds (an upper
        estimate from the widest block), so that the engine can leave room for them."""
        act = 2 if self.dtype == torch.bfloat16 else 4
        widest = max((b.scratch_elements_per_token() for b in self.blocks), default=0)
        H = self.spec.hidden_size
        H4 = 8 * H if self.readds_embedding else 4 * H
        return tokens * (H4 + widest * act) + wanted * (self.spec.vocab_size * 4 + H * act)


register_model("decoder", DecoderModel)
