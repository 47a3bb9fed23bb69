"""A decoder put together from parts, and the order in which its layers run.

``DecoderModel`` holds an embedding, a list of blocks, a final norm and a head.
The order of execution is data: ``schedule`` is a list of ``LayerCall``; a call
names the block to run and the call whose cache it uses.  By default call i runs
block i on a cache of its own.  A schedule may name a block twice (each call
that owns a cache gets its own), or let a call read the cache an earlier call
wrote (the reference's ``kv_src`` layers, ``lua/lgml/transformer.lua:1829-1830``,
``:592``).  mischief/lgml's loop over layers is ``M:forward``
(``:2285-2365``): embedding (``:2303``), the layers (``:2312-2345``), the rows
whose logits are wanted (``:2349-2350``), the final norm and the head
(``:2095-2096``).
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence

import torch

from .. import ops
from ..parts.norm import PendingDelta, ScaledTerms, UnitMix
from ..parts.streams import PendingStreams
from ..weights import VECTOR, TensorSpec


@dataclass(frozen=True)
class LayerCall:
    block: int                    # index into DecoderModel.blocks
    cache: Optional[int] = None   # index of the call that owns the cache used; None = this call
    add_input: bool = False       # the residual stream as it was before the first call is added to it before this call
    add_row: Optional[int] = None  # this row of the model's table of pass vectors is added to every token's x before this call
    begins_pass: Optional[int] = None  # this pass of a loop begins here: the model's ``pass_input`` makes x anew before this call


class DecoderModel:
    def __init__(self, config, embedding, blocks, final_norm, head, schedule: Optional[List[LayerCall]] = None,
                 block_prefix: str = "model.layers.{}", final_norm_prefix: str = "model.norm",
                 embed_scale: Optional[float] = None, logit_scale: Optional[float] = None, logit_softcap: Optional[float] = None,
                 ignored_tensors: Sequence[str] = (), embed_norm=None, embed_norm_prefix: str = "model.embed_norm",
                 delta_dtype: Optional[torch.dtype] = None, pass_rows: Optional[str] = None, streams: int = 0,
                 pass_input=None, step_parts: Sequence = ()):
        self.config = config
        # the residual in this many streams (``parts/streams.py``; the blocks and the final norm are made for them); 0: one x
        self.streams = int(streams)
        # the type in which mixers and feed-forwards hand their results to the residual stream (None: the compute type)
        self.delta_dtype = delta_dtype
        # the name of a tensor [rows, width] whose rows schedule entries add to x (``LayerCall.add_row``)
        self.pass_rows_name, self.pass_rows = pass_rows, None
        # what makes x anew at the start of a pass (``LayerCall.begins_pass``; ``parts/token_mix.py``: ``PassInput``)
        self.pass_input = pass_input
        # things with ``begin(rt, batch)`` that settle something for the whole step before its first layer
        self.step_parts = tuple(step_parts)
        self.embedding = embedding
        self.blocks = list(blocks)
        self.final_norm = final_norm
        self.head = head
        self.block_prefix = block_prefix
        self.final_norm_prefix = final_norm_prefix
        # a norm between the embedding and the first layer (None: the rows themselves are the residual stream)
        self.embed_norm, self.embed_norm_prefix = embed_norm, embed_norm_prefix
        # name patterns of tensors that a folder of this architecture may carry unread
        self.ignored_tensors = tuple(ignored_tensors)
        # scales that other families of the reference apply and Llama does not (None = no kernel):
        # on the embedding's rows (``embd_scale``, ``lua/lgml/transformer.lua:2303-2306``), on the
        # logits, and the logits' cap (``logit_scale``, ``softcap``, ``:2097-2102``)
        self.embed_scale, self.logit_scale, self.logit_softcap = embed_scale, logit_scale, logit_softcap
        self.schedule = list(schedule) if schedule is not None else [LayerCall(i) for i in range(len(self.blocks))]
        for ci, call in enumerate(self.schedule):
            if not 0 <= call.block < len(self.blocks):
                raise ValueError(f"schedule entry {ci} names block {call.block}, but there are {len(self.blocks)}")
            if call.cache is not None:
                if not 0 <= call.cache < ci:
                    raise ValueError(f"schedule entry {ci} reads the cache of entry {call.cache}, which does not run before it")
                if self.schedule[call.cache].cache is not None:
                    raise ValueError(f"schedule entry {ci} reads the cache of entry {call.cache}, which has none of its own")
            if call.add_row is not None and pass_rows is None:
                raise ValueError(f"schedule entry {ci} adds a pass vector, but the model names no table of them")
            if call.begins_pass is not None and ci == 0 and embed_norm is not None:
                raise ValueError("a pass that starts the model reads the embedding's rows, not a norm of them")
            if call.begins_pass is not None and (pass_input is None or self.streams):
                raise ValueError(f"schedule entry {ci} begins a pass, but the model has no part that makes x anew")
            if self.streams and (call.add_row is not None or call.add_input):
                raise ValueError(f"schedule entry {ci} adds a row to x, which is {self.streams} streams")
        self.n_pass_rows = 1 + max((call.add_row for call in self.schedule if call.add_row is not None), default=-1)
        self.vocab_size = head.vocab
        parts = [embedding, final_norm, head] + self.blocks + [p for p in (embed_norm, pass_input) if p is not None]
        self.graph_safe = all(getattr(p, "graph_safe", False) for p in parts)
        self.max_position = getattr(config, "max_position_embeddings", None)

    # ---- weights -----------------------------------------------------------------------
    def tensor_specs(self) -> List[TensorSpec]:
        specs = list(self.embedding.tensor_specs(""))
        if self.embed_norm is not None:
            specs += self.embed_norm.tensor_specs(self.embed_norm_prefix)
        for i, b in enumerate(self.blocks):
            specs += b.tensor_specs(self.block_prefix.format(i))
        if self.pass_input is not None:
            specs += self.pass_input.tensor_specs("")
        specs += self.final_norm.tensor_specs(self.final_norm_prefix)
        specs += self.head.tensor_specs("")
        if self.pass_rows_name is not None and self.n_pass_rows:
            specs.append(TensorSpec(self.pass_rows_name, (self.n_pass_rows, self.embedding.width), VECTOR))
        seen = {}
        for s in specs:          # a tensor two parts share (e.g. frequency factors) is listed once
            seen.setdefault(s.name, s)
        return list(seen.values())

    def bind(self, tensors: Dict[str, torch.Tensor], rt) -> None:
        self.embedding.bind("", tensors, rt)
        if self.embed_norm is not None:
            self.embed_norm.bind(self.embed_norm_prefix, tensors, rt)
        for i, b in enumerate(self.blocks):
            b.bind(self.block_prefix.format(i), tensors, rt)
        if self.pass_input is not None:
            self.pass_input.bind("", tensors, rt)
        self.final_norm.bind(self.final_norm_prefix, tensors, rt)
        self.head.bind("", tensors, rt)
        if self.pass_rows_name is not None and self.n_pass_rows:
            self.pass_rows = tensors[self.pass_rows_name].float().contiguous()

    # ---- cache -------------------------------------------------------------------------
    def cache_layout(self) -> Dict[int, object]:
        """schedule index -> the cache spec of the calls that own a cache."""
        out = {}
        for ci, call in enumerate(self.schedule):
            if call.cache is None:
                spec = self.blocks[call.block].cache_spec()
                if spec is not None:
                    out[ci] = spec
        return out

    @staticmethod
    def _with_row(x, pending, row, block):
        """What is pending for x once ``row`` is to be added to every token's x as well: a block whose first norm takes
        such a delta gets it with the row; for any other the sums are made here."""
        if getattr(block, "takes_pending_row", False) and (pending is None or (isinstance(pending, PendingDelta) and pending.row_add is None)):
            return dataclasses.replace(pending, row_add=row) if pending is not None else PendingDelta(row_add=row)
        DecoderModel._fold(x, pending)
        ops.sandwich_norm(x, None, 0.0, None, row_add=row)
        return None

    @staticmethod
    def _fold(x, pending) -> None:
        """x += what is pending, now, by a kernel of its own."""
        if isinstance(pending, ScaledTerms):
            ops.scaled_norm(x, pending.terms, keep=pending.keep)
        elif isinstance(pending, PendingDelta):
            d = pending.delta
            if isinstance(d, UnitMix):
                ops.sandwich_norm(x, None, pending.eps, None, delta=(d.a, d.b), units=(d.u_a, d.u_b), w_post=pending.w_post, row_add=pending.row_add)
            else:
                ops.sandwich_norm(x, None, pending.eps, None, delta=d.sum() if isinstance(d, ops.Partials) else d, w_post=pending.w_post,
                                  row_add=pending.row_add)
        elif pending is not None:
            ops.residual_fold(x, pending)

    # ---- the forward pass of one step --------------------------------------------------
    def forward(self, rt, batch) -> torch.Tensor:
        """float32 logits [len(batch.logit_rows), vocab] for the tokens of ``batch``."""
        for part in self.step_parts:
            part.begin(rt, batch)
        # a pass that starts the model reads the embedding itself
        starts = self.schedule[0].begins_pass is not None
        if starts:
            x = torch.empty((batch.token_ids.numel(), self.embedding.width), dtype=torch.float32, device=batch.token_ids.device)
        else:
            x = self.embedding.forward(rt, batch.token_ids)
        if self.embed_scale is not None and not starts and not (self.streams and self.embed_norm is None):
            ops.scale_cap(x, self.embed_scale)
        if self.embed_norm is not None:
            x = self.embed_norm.forward(rt, x, torch.float32)
        rt.delta_dtype = self.delta_dtype
        x_in = x.clone() if any(call.add_input for call in self.schedule) else None
        pending = None
        if self.streams:        # the first norm's kernel makes the streams from the (scaled) rows
            pending = PendingStreams(start=x, start_scale=self.embed_scale if self.embed_scale is not None and self.embed_norm is None else 1.0)
            x = torch.empty((x.shape[0], self.streams, x.shape[1]), dtype=torch.float32, device=x.device)
        for ci, call in enumerate(self.schedule):
            if call.add_input:
                if pending is not None:
                    self._fold(x, pending)
                    pending = None
                ops.residual_fold(x, x_in)
            if call.begins_pass is not None:
                pending = self.pass_input.forward(rt, x, pending, batch, call.begins_pass, starts_model=ci == 0)
            if call.add_row is not None:
                pending = self._with_row(x, pending, self.pass_rows[call.add_row], self.blocks[call.block])
            owner = ci if call.cache is None else call.cache
            cache = batch.cache_view(owner, writable=call.cache is None)
            x, pending = self.blocks[call.block].forward(rt, x, pending, batch, cache)
        h = self.final_norm.forward(rt, x, rt.dtype, delta=pending, rows=batch.logit_rows)
        logits = self.head.forward(rt, h)
        if self.logit_scale is not None or self.logit_softcap:
            ops.scale_cap(logits, 1.0 if self.logit_scale is None else self.logit_scale, self.logit_softcap or 0.0)
        return logits
