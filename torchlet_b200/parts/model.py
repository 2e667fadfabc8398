"""A model put together from a ``ModelSpec``: embedding, the layers run in the order
of the schedule, final norm, LM head (embedding -> blocks -> norm -> head,
v10_triton_paged_gqa/model/qwen2_5.py:21-87).  It knows no architecture by name.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from ..config.spec import ModelSpec
from .base import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, TOKEN_INPUTS, KVSpec, StateSpec, TensorSpec, build_part
from .linear import Linear


@dataclass
class ExecutionCacheNeed:
    """What one schedule entry keeps between steps."""

    entry: int
    owner: int  # the entry whose cache is used (itself unless cache_from is set)
    kv: Optional[KVSpec]
    state: object  # the mixer's: None, a StateSpec, or a dict name -> StateSpec
    block_state: object = None  # the block arrangement's own, in the same forms


def _layer_parts(layer) -> list:
    """(registry, part description, full tensor-name prefix, role) of every part of a layer, in the
    order their tensors are listed and loaded.  The names come from the layer's description."""
    parts = [(NORMS, slot.part, layer.prefix + slot.prefix, slot.role) for slot in layer.norms]
    parts.insert(min(1, len(parts)), (MIXERS, layer.mixer, layer.prefix + layer.mixer_prefix, "mixer"))
    if layer.feed_forward is not None:
        parts.append((FEED_FORWARDS, layer.feed_forward, layer.prefix + layer.feed_forward_prefix, "feed_forward"))
    if layer.token_input is not None:
        parts.append((TOKEN_INPUTS, layer.token_input, layer.prefix + layer.token_input_prefix, "token_input"))
    return parts


def expected_tensors(spec: ModelSpec) -> list[TensorSpec]:
    """Every tensor the checkpoint must hold, by name, with its shape."""
    out = [TensorSpec(spec.embedding_name, (spec.vocab_size, spec.hidden_size))]
    if spec.token_pairs is not None:
        out.append(TensorSpec(spec.token_pairs.table_name, (spec.token_pairs.buckets + 1, spec.hidden_size)))
    if spec.stream_rows_name is not None:
        out.append(TensorSpec(spec.stream_rows_name, (spec.stream_rows, spec.hidden_size)))
    if spec.embedding_norm is not None:
        out += NORMS.get(spec.embedding_norm.kind).expected_tensors(spec.embedding_norm, spec.embedding_norm_prefix)
    for layer in spec.layers:
        for registry, part, prefix, _ in _layer_parts(layer):
            out += registry.get(part.kind).expected_tensors(part, prefix)
        out += BLOCKS.get(layer.block).expected_tensors(layer)
    out += NORMS.get(spec.final_norm.kind).expected_tensors(spec.final_norm, spec.final_norm_prefix)
    out.append(TensorSpec(spec.lm_head_name, (spec.vocab_size, spec.hidden_size), optional=spec.tie_word_embeddings))
    unique, seen = [], set()
    for want in out:  # a tensor several parts share (a table all layers cut their part from) is listed once
        if want.name not in seen:
            seen.add(want.name)
            unique.append(want)
    return unique


class LayeredModel:
    def __init__(self, spec: ModelSpec):
        spec.validate()
        self.spec = spec
        self.blocks = []
        for layer in spec.layers:
            block_cls = BLOCKS.get(layer.block)
            missing = [role for role in block_cls.norm_roles if role not in {slot.role for slot in layer.norms}]
            if missing:
                raise ValueError(f"layer {layer.prefix!r}: the arrangement {layer.block!r} needs norms for {missing}")
            self.blocks.append(
                block_cls(
                    build_part(MIXERS, layer.mixer),
                    build_part(FEED_FORWARDS, layer.feed_forward) if layer.feed_forward is not None else None,
                    {slot.role: build_part(NORMS, slot.part) for slot in layer.norms},
                    **({"params": layer.block_params} if layer.block_params else {}),
                    **({"token_input": build_part(TOKEN_INPUTS, layer.token_input)} if layer.token_input is not None else {}),
                )
            )
        self.final_norm = build_part(NORMS, spec.final_norm)
        self.embedding_norm = build_part(NORMS, spec.embedding_norm) if spec.embedding_norm is not None else None
        self.embedding: torch.Tensor | None = None
        self.pair_table: torch.Tensor | None = None  # [buckets + 1, hidden], see ``TokenPairs``
        self.stream_rows: torch.Tensor | None = None  # [rows, hidden] float32, see ``ScheduleEntry.add_row``
        self.lm_head: Linear | None = None
        self.dtype: torch.dtype | None = None
        self.device = None

    # ------------------------------------------------------------ structure
    def cache_needs(self) -> list[ExecutionCacheNeed]:
        needs = []
        for i, entry in enumerate(self.spec.schedule):
            mixer = self.blocks[entry.layer].mixer
            owner = i if entry.cache_from is None else entry.cache_from
            if entry.cache_from is not None:
                theirs = self.blocks[self.spec.schedule[owner].layer].mixer.kv_spec()
                mine = mixer.kv_spec()
                if theirs is None or mine is None or (theirs.num_kv_heads, theirs.head_dim, theirs.planes) != (mine.num_kv_heads, mine.head_dim, mine.planes):
                    raise ValueError(f"schedule entry {i} cannot read the cache of entry {owner}: shapes differ")
            needs.append(ExecutionCacheNeed(i, owner, mixer.kv_spec(), mixer.state_spec(),
                                            self.blocks[entry.layer].state_spec()))
        return needs

    def state_specs(self) -> dict:
        """What the model itself keeps per live request (name -> ``StateSpec``; ``ctx.model_state`` holds the tensors)."""
        return {"last_token": StateSpec((1,), "int32")} if self.spec.token_pairs is not None else {}

    # --------------------------------------------------------------- weights
    def load(self, tensors: dict, device, dtype: torch.dtype) -> None:
        """Lay the checkpoint's tensors (by name) out on the device for the kernels."""
        spec = self.spec
        self.device, self.dtype = torch.device(device), dtype
        self.embedding = tensors[spec.embedding_name].to(device=device, dtype=dtype).contiguous()
        if spec.token_pairs is not None:
            self.pair_table = tensors[spec.token_pairs.table_name].to(device=device, dtype=dtype).contiguous()
        if spec.stream_rows_name is not None:
            self.stream_rows = tensors[spec.stream_rows_name].to(device=device, dtype=torch.float32).contiguous()
        for layer, block in zip(spec.layers, self.blocks):
            for _, _, prefix, role in _layer_parts(layer):
                part = {"mixer": block.mixer, "feed_forward": block.feed_forward,
                        "token_input": getattr(block, "token_input", None)}.get(role) or block.norms[role]
                part.load(tensors, prefix, device, dtype)
            block.load(tensors, layer, device, dtype)
        self.final_norm.load(tensors, spec.final_norm_prefix, device, dtype)
        if self.embedding_norm is not None:
            self.embedding_norm.load(tensors, spec.embedding_norm_prefix, device, dtype)
        if spec.tie_word_embeddings:
            self.lm_head = Linear.from_device_weight(self.embedding)
        else:
            self.lm_head = Linear(tensors[spec.lm_head_name], None, device, dtype)

    # --------------------------------------------------------------- forward
    def forward(self, ctx, caches: list) -> torch.Tensor:
        """Run the step's tokens through the schedule; returns the float32 stream [T, hidden]."""
        shape = (ctx.num_tokens, self.spec.hidden_size)
        acc = ctx.buffer("stream", shape, torch.float32)
        streams = self.spec.streams
        z = None
        if streams is not None:
            z = ctx.buffer("streams", (ctx.num_tokens, streams, self.spec.hidden_size), torch.float32)
        again = any(entry.add_embedding for entry in self.spec.schedule)
        first = ctx.buffer("stream.first", shape, torch.float32) if again else None  # the embedding output, kept
        if self._embeds_at_once():
            self._embed_at_once(ctx, acc if streams is None else z)
            if again:
                first.copy_(acc)
        else:
            self._embed(ctx, acc, first)
            if streams is not None:
                ops.hyper_fanout(acc, z)
        if streams is None:
            for i, entry in enumerate(self.spec.schedule):
                if entry.add_embedding:
                    ctx.flush_pending()
                    ops.scaled_add(acc, first, 1.0)
                if entry.add_row is not None:
                    ctx.add_row(acc, self.stream_rows[entry.add_row])
                self.blocks[entry.layer].forward(ctx, acc, caches[i])
            ctx.flush_pending()
            return acc
        # several residual streams a token, all equal to the embedding at the start; their sum at the end
        for i, entry in enumerate(self.spec.schedule):
            self.blocks[entry.layer].forward(ctx, z, caches[i])
        write = ctx.take_write(z)  # the last sub-layer's, joined with the sum
        ctx.flush_pending()
        ops.hyper_collapse(z, acc, write)
        return acc

    def _embeds_at_once(self) -> bool:
        """Whether token row, pair row, norm and the copies to the streams run as one kernel: a model with a pair table
        (its norm, if it has one, must be over whole rows)."""
        if self.spec.token_pairs is None:
            return False
        if self.embedding_norm is not None and self.embedding_norm.residual_terms() is None:
            raise ValueError("a table of token pairs is not built together with a grouped norm of the embedding")
        return True

    def _embed_at_once(self, ctx, out) -> None:
        pairs = self.spec.token_pairs
        norm = self.embedding_norm.residual_terms() if self.embedding_norm is not None else None
        ops.token_embed(self.embedding, ctx.tokens, out, scale=self.spec.embedding_scale,
                        pairs=(self.pair_table, pairs.mul_prev, pairs.mul_cur), norm=norm,
                        ctx_arrays=(ctx.positions, ctx.token_req, ctx.req_indptr, ctx.slots), last=ctx.model_state["last_token"])

    def _embed(self, ctx, acc, first) -> None:
        """The embedding output into ``acc`` (and into ``first``, if that is kept)."""
        if self.embedding_norm is None:
            ops.embed(self.embedding, ctx.tokens, acc, self.spec.embedding_scale)
            if first is not None:
                ops.embed(self.embedding, ctx.tokens, first, self.spec.embedding_scale)
            return
        # the norm writes float32 rows: the stream stays 32-bit from its first value on
        raw = ctx.buffer("stream.embedding", tuple(acc.shape), torch.float32)
        ops.embed(self.embedding, ctx.tokens, raw, self.spec.embedding_scale)
        self.embedding_norm.apply(ctx, raw, out=acc)
        if first is not None:
            self.embedding_norm.apply(ctx, raw, out=first)

    def logits(self, ctx, acc: torch.Tensor, rows: torch.Tensor, out: torch.Tensor) -> None:
        """Float32 logits of the stream rows ``rows`` (int32) into ``out`` [len(rows), vocab]."""
        x = self.final_norm.apply(ctx, acc, rows=rows, name="final.normed")
        self.lm_head.forward(x, out)
        if self.spec.logit_scale != 1.0:
            ops.scale_(out, self.spec.logit_scale)
