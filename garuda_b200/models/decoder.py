"""A decoder as data: an embedding, a list of layers, the order in which they
run, a final norm and an output head.

The reference's stack is a fixed loop (garuda/src/llama/mod.rs:1092-1095,
:1183-1188); here the order is a list of ``LayerCall``. A layer may be called
twice, and a call may read the cache that an earlier call filled instead of
keeping one of its own. Nothing in this file knows an architecture: an
architecture is a function from its configuration to a ``ModelSpec``
(``garuda_b200/models/llama.py`` is the one there is).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from ..parts.base import (PartSpec, TensorSpec, PagedKV, PagedLatent, FixedState, LayerCache, build_part,
                          tensor_name, _REGISTRIES)
from ..parts.block import BlockSpec, NormedInput


@dataclass(frozen=True)
class LayerCall:
    """One entry of the run order. ``layer`` indexes ``ModelSpec.layers``.
    ``reads_cache_of``: index of an earlier entry of the run order whose cache
    this call reads (it then stores nothing itself). A model that runs a stretch of its layers
    several times marks the first call of every pass: ``add_embedding`` adds the embedding's
    output (the stream as it was before the first layer) to the stream before the call, or
    ``mix_embedding`` names a model-level ``[width, 2 width]`` matrix ``W`` and the stream becomes ``W [stream;
    embedding's output]``; ``add_row = (tensor, r)`` then adds row ``r`` of that model-level ``[rows, width]`` tensor."""
    layer: int
    reads_cache_of: Optional[int] = None
    add_embedding: bool = False
    mix_embedding: Optional[str] = None
    add_row: Optional[Tuple[str, int]] = None


@dataclass
class ModelSpec:
    architecture: str
    width: int
    vocab_size: int
    max_positions: int
    embedding: str                       # tensor name of the [vocab, width] table
    layers: List[BlockSpec]
    order: List[LayerCall]
    final_norm: PartSpec
    head: Optional[str]                  # tensor name of the [vocab, width] head; None: tied
    embedding_init: Tuple = ("normal", 0.02)
    embedding_scale: float = 1.0         # the embedding's output is the table's row times this
    embedding_norm: Optional[PartSpec] = None    # ... and then an RMS norm of it
    # the residual as several streams [T, streams, width], all equal to the embedding's output at the
    # start, summed before the final norm; None: one residual [T, width]
    streams: Optional[int] = None
    logit_scale: float = 1.0             # logits = head(x) * logit_scale ...
    logit_softcap: Optional[float] = None   # ... then c * tanh(logits / c)
    # tensors of the model itself that no part owns (what ``LayerCall.add_row`` and ``mix_embedding`` name): name -> spec
    extra_tensors: Optional[Dict[str, TensorSpec]] = None
    eos_token_ids: Tuple[int, ...] = ()  # generation ends on any of them (config.json may list several)
    # names a model folder may hold although the model reads nothing from them (a tied model's
    # stored copy of its head); anything else the model did not ask for is an error
    ignored_tensors: Tuple[str, ...] = ()

    @property
    def eos_token_id(self) -> Optional[int]:
        return self.eos_token_ids[0] if self.eos_token_ids else None


@dataclass(frozen=True)
class CacheGroup:
    """Calls of the run order whose caches have the same needs and therefore
    share a pool of pages and a block table."""
    need: object                         # PagedKV
    calls: Tuple[object, ...]            # cache keys: indices into ModelSpec.order (calls that write), or (index, member)


class Decoder:
    def __init__(self, spec: ModelSpec):
        self.spec = spec
        self.blocks = [_REGISTRIES["block"][b.arrangement](b) for b in spec.layers]
        self.final_norm = build_part("norm", spec.final_norm)
        self.embedding_norm = build_part("norm", spec.embedding_norm) if spec.embedding_norm else None
        if self.embedding_norm is not None and (not hasattr(self.embedding_norm, "fold") or spec.embedding_scale != 1.0 or spec.streams is not None):
            raise ValueError("an embedding that is normed takes an RMS norm, no scale and one stream")
        self.ops = None
        self.dtype = None
        # cache needs of the run order
        self.call_need = []
        for i, call in enumerate(spec.order):
            if not 0 <= call.layer < len(self.blocks):
                raise ValueError(f"run order entry {i} names layer {call.layer}, but there are {len(self.blocks)}")
            need = self.blocks[call.layer].mixer.cache_need()
            if call.reads_cache_of is not None:
                src = call.reads_cache_of
                if not 0 <= src < i or spec.order[src].reads_cache_of is not None:
                    raise ValueError(f"run order entry {i} must read the cache of an earlier entry that keeps one")
                if self.call_need[src] != need:
                    raise ValueError(f"run order entry {i} reads a cache of another shape: {self.call_need[src]} vs {need}")
            self.call_need.append(need)
        # A cache key is the index of a run-order entry, or (index, member) for a mixer that is made
        # of several mixers with a cache or a state each.
        groups: Dict[object, List[object]] = {}
        self.state_calls: List[object] = []
        for i, (call, need) in enumerate(zip(spec.order, self.call_need)):
            if call.reads_cache_of is not None or need is None:
                continue
            members = [(i, need)] if not isinstance(need, tuple) else [((i, k), n) for k, n in enumerate(need)]
            for key, n in members:
                if n is None:
                    continue
                if isinstance(n, (PagedKV, PagedLatent)):
                    groups.setdefault(n, []).append(key)
                elif isinstance(n, FixedState):
                    self.state_calls.append(key)
                else:
                    raise TypeError(f"unknown cache need {n!r}")
        self.cache_groups = [CacheGroup(need, tuple(calls)) for need, calls in groups.items()]

    def need_at(self, key):
        """The cache need behind a cache key: of a run-order entry, or of one member of its mixer."""
        if isinstance(key, tuple):
            return self.call_need[key[0]][key[1]]
        return self.call_need[key]

    @property
    def graph_safe(self) -> bool:
        """Whether a decode step of this model may be captured in a CUDA graph: every part says so."""
        return all(b.graph_safe for b in self.blocks) and all(norm.graph_safe for norm, _ in self._model_norms())

    # ---- tensors ---------------------------------------------------------
    def expected_tensors(self) -> Dict[str, TensorSpec]:
        s = self.spec
        out = {s.embedding: TensorSpec((s.vocab_size, s.width), init=s.embedding_init)}
        for block in self.blocks:
            for part, prefix in block.parts():
                for local, ts in part.tensors().items():
                    out[tensor_name(prefix, local)] = ts
        for norm, ns in self._model_norms():
            for local, ts in norm.tensors().items():
                out[tensor_name(ns.prefix, local)] = ts
        out.update(s.extra_tensors or {})
        if s.head is not None:
            out[s.head] = TensorSpec((s.vocab_size, s.width), init=s.embedding_init)
        return out

    def _model_norms(self):
        """The norms that belong to no layer, with their specs."""
        pairs = [(self.final_norm, self.spec.final_norm), (self.embedding_norm, self.spec.embedding_norm)]
        return [(norm, ns) for norm, ns in pairs if norm is not None]

    def load(self, tensors: Dict[str, torch.Tensor], ops, dtype: torch.dtype) -> None:
        """``tensors``: every name of ``expected_tensors()`` on the device."""
        s = self.spec
        self.ops, self.dtype = ops, dtype
        self.embedding = tensors[s.embedding]
        self.head = self.embedding if s.head is None else tensors[s.head]
        for block in self.blocks:
            for part, prefix in block.parts():
                part.load({local: tensors[tensor_name(prefix, local)] for local in part.tensors()}, ops, dtype)
        for norm, ns in self._model_norms():
            norm.load({local: tensors[tensor_name(ns.prefix, local)] for local in norm.tensors()}, ops, dtype)
        self.extra = {name: tensors[name].contiguous() for name in (s.extra_tensors or {})}
        self.rows32 = {call.add_row: self.extra[call.add_row[0]][call.add_row[1]].float().contiguous()
                       for call in s.order if call.add_row is not None}
        self.keeps_embedding = any(call.add_embedding for call in s.order)
        self.mixes_embedding = any(call.mix_embedding is not None for call in s.order)

    # ---- one step ----------------------------------------------------------
    def forward(self, ctx, layer_caches: List[Optional[LayerCache]]) -> torch.Tensor:
        """Runs the batch of ``ctx`` through the run order and returns 32-bit
        logits ``[W, vocab]`` for the batch's ``logit_rows`` only: the final norm
        and the head touch no other row (garuda/src/llama/mod.rs:1110-1113)."""
        b, ops, s = ctx.batch, self.ops, self.spec
        if s.streams is not None:
            return self._forward_streams(ctx, layer_caches)
        x = ctx.ws.get("residual", (b.num_tokens, s.width), torch.float32)
        # the operand [stream; embedding's output] of a mix, in the compute dtype
        pair = ctx.ws.get("embedding_pair", (b.num_tokens, 2 * s.width), ctx.dtype) if self.mixes_embedding else None
        if self.embedding_norm is not None:
            ops.embedding_norm(self.embedding, b.token_ids, *self.embedding_norm.fold(), x, pair)
        elif s.embedding_scale != 1.0:
            ops.embedding(self.embedding, b.token_ids, x, s.embedding_scale)
        else:
            ops.embedding(self.embedding, b.token_ids, x)
        if pair is not None and self.embedding_norm is None:
            ops.residual_norm(x, out=pair[:, s.width:])
        x0 = None
        if self.keeps_embedding:
            x0 = ctx.ws.get("embedding_out", (b.num_tokens, s.width), torch.float32)
            x0.copy_(x)
        # a layer's last product may fold in the first half of the next layer's norm
        pending = None
        for i, call in enumerate(s.order):
            block = self.blocks[call.layer]
            if call.mix_embedding is not None:
                pending = self._mix_embedding(ctx, x, pair, call, block, rounded=pending is not None or (i == 0 and self.embedding_norm is not None))
            elif call.add_embedding or call.add_row is not None:
                row = self.extra[call.add_row[0]][call.add_row[1]] if call.add_row is not None else None
                ops.residual_axpy(x, x0 if call.add_embedding else None, 1.0, row)
            nxt = self.blocks[s.order[i + 1].layer] if i + 1 < len(s.order) else None
            if nxt is not None and s.order[i + 1].mix_embedding is not None:
                # the mix in front of the next layer wants the stream rounded, beside the embedding's output
                next_norm = NormedInput(out=pair[:, :s.width]) if getattr(block, "writes_normed_input", False) else None
            else:
                takes = getattr(nxt, "takes_pending_norm", None)
                next_norm = takes(ops) if takes is not None else None
            if pending is not None or next_norm is not None:
                pending = block.forward(ctx, x, layer_caches[i], pending=pending, next_norm=next_norm)
            else:
                pending = block.forward(ctx, x, layer_caches[i])
            if ctx.layer_probe is not None:
                ctx.layer_probe(i, x)
        return self._logits(ctx, x)

    def _mix_embedding(self, ctx, x, pair, call, block, rounded):
        """``x <- W [x; embedding's output] + row`` before a layer call. ``rounded``: the pass in front has left ``x``
        in ``pair``. Returns the layer's normed input where the layer takes one from a pass over the residual."""
        ops, width = self.ops, self.spec.width
        if not rounded:
            ops.residual_norm(x, out=pair[:, :width])
        ops.linear(pair, self.extra[call.mix_embedding], x)
        row = self.rows32.get(call.add_row)
        takes = getattr(block, "takes_pending_norm", None)
        wanted = takes(ops) if takes is not None else None
        if isinstance(wanted, NormedInput):
            weight, eps, out = wanted.into(ctx, x, 1)
            ops.residual_norm(x, row=row, then_weight=weight, then_eps=eps, out=out)
            return out
        if row is not None:
            ops.residual_axpy(x, None, 1.0, row)
        return None

    def _logits(self, ctx, x) -> torch.Tensor:
        b, ops, s = ctx.batch, self.ops, self.spec
        w = b.num_logit_rows
        logits = ctx.ws.get("logits", (w, s.vocab_size), torch.float32)
        if w:
            z = self.final_norm.forward(ctx, x, rows=b.logit_rows, out_name="final_normed")
            ops.linear(z, self.head, logits)
            if s.logit_scale != 1.0 or s.logit_softcap:
                ops.scale_softcap(logits, s.logit_scale, s.logit_softcap or 0.0)
        return logits

    def _forward_streams(self, ctx, layer_caches) -> torch.Tensor:
        """The run order over a residual of several streams. A layer's last write to the streams
        computes the next layer's first normed input in the same pass where the kernels can."""
        b, ops, s = ctx.batch, self.ops, self.spec
        if any(call.add_embedding or call.mix_embedding is not None or call.add_row is not None for call in s.order):
            raise ValueError("a residual of several streams takes no additions between layer calls")
        x = ctx.ws.get("residual", (b.num_tokens, s.streams, s.width), torch.float32)
        ops.embedding(self.embedding, b.token_ids, x, s.embedding_scale)
        normed = None
        for i, call in enumerate(s.order):
            block = self.blocks[call.layer]
            nxt = self.blocks[s.order[i + 1].layer] if i + 1 < len(s.order) else None
            then = nxt.first_read() if nxt is not None and ctx.layer_probe is None else None
            normed = block.forward(ctx, x, layer_caches[i], normed=normed, then=then)
            if ctx.layer_probe is not None:
                ctx.layer_probe(i, x)
        return self._logits(ctx, x)
