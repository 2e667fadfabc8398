"""Choice of the kernels of an attention whose scores may be mixed across the heads and whose window may keep the
sequence's first tokens.

``query_form``: how csrc/qkv_prepare.cu is to write the queries of mixed scores (its ``spread``): 1, spread over all KV
heads, for the kernels that take one dot product over all of a token's keys.
"""
from __future__ import annotations


def query_form(mixer, ctx, cache) -> int:
    return 1


def forward(mixer, ctx, q, cache, out, spread: int) -> bool:
    """False: no tensor-core kernel takes the sizes; the caller uses the one-warp-a-row kernel."""
    return False
