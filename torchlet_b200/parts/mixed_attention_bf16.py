"""Choice and planning of the bfloat16 tensor-core kernels of an attention whose scores may be mixed across the heads and
whose window may keep the sequence's first tokens.

Requests that bring a portion of a prompt run on the tcgen05 kernel (csrc/attention_spread.cu) in tiles of 128 packed rows
planned on the host; with mixed scores it wants the queries spread over all KV heads.  Requests that bring a single token
run on the ``mma.sync`` kernel that holds all heads' scores of a key at once and mixes them itself
(csrc/attention_mixed_decode.cu); it wants the queries as they are.  A step whose sizes one of the two does not take runs
on the one-warp-a-row kernel (csrc/attention_generic.cu), with spread queries throughout.
"""
from __future__ import annotations

import torch

from .. import ops
from . import attention_bf16


def _kinds(ctx) -> tuple:
    """(whether a request of the step brings a single token, whether one brings several)."""
    if ctx.decode_only:
        return True, False
    lens = ctx.req_indptr_host[1:] - ctx.req_indptr_host[:-1]
    return bool((lens == 1).any()), bool((lens > 1).any())


def usable(mixer, ctx, cache) -> bool:
    if ctx.dtype != torch.bfloat16:
        return False
    single, several = _kinds(ctx)
    H, G, P = mixer.num_heads, mixer.num_kv_heads, mixer.head_dim
    if several and not ops.attention_spread_supported(P, H // G, cache.page_size, mixer.scale):
        return False
    return not single or ops.attention_mixed_decode_tile(H, G, P, cache.page_size, mixer.v_dim) > 0


def query_form(mixer, ctx, cache) -> int:
    """How csrc/qkv_prepare.cu is to write the queries of mixed scores (its ``spread``)."""
    if not usable(mixer, ctx, cache):
        return 1
    single, several = _kinds(ctx)
    return 2 if single and several else (1 if several else 0)


def decode_splits(requests: int, keys: int, device) -> int:
    """CTAs that share the key tiles of one request: as many as fill one wave (the kernel's stages leave room for one CTA an
    SM), no share below 96 keys.  ``keys``: the most keys a request of the step, or of the captured graph, may see."""
    index = torch.cuda.current_device() if device.index is None else device.index
    return max(1, min(attention_bf16._sm_count(index) // max(1, requests), -(-keys // 96)))


def forward(mixer, ctx, q, cache, out) -> bool:
    """``q``: rows as ``query_form`` asked for.  False: the caller uses the one-warp-a-row kernel."""
    if not usable(mixer, ctx, cache):
        return False
    H, G, P = mixer.num_heads, mixer.num_kv_heads, mixer.head_dim
    common = dict(nh=H, nkv=G, p_size=P, page_size=cache.page_size, window=mixer.window, keep=mixer.keep_first,
                  v_cols=mixer.v_dim, scale=mixer.scale)
    plan = attention_bf16._plan(ctx, H // G, ops.attention_spread_rows(H // G))
    if plan["prefill"] is not None:
        tile_req, tile_row, count = plan["prefill"]
        ops.attention_spread(q, cache.pages, cache.block_table, ctx.req_indptr, ctx.kv_before, tile_req, tile_row, count, out,
                             spread=mixer.score_mix, **common)
    if plan["decode"] is not None:
        tile_req, count = plan["decode"]
        seen = ctx.max_kv_len
        if mixer.window:  # the window's keys, the kept ones and the ends of their tiles
            seen = min(seen, mixer.window + mixer.keep_first + 128)
        ops.attention_mixed_decode(q, cache.pages, cache.block_table, ctx.req_indptr, ctx.kv_before, tile_req, count, out,
                                   talk=mixer.talk, splits=decode_splits(count, seen, q.device), **common)
    return True
