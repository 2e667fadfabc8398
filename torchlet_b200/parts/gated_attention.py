"""Grouped-query attention over a paged cache with the options newer designs combine:

* ``qk_norm`` "whole": q and k are RMS-normed over the WHOLE projection (all heads at once, plain
  weights ``q.norm`` / ``k.norm``) before the rotation; None: no norm;
* ``values_from_keys``: there is no value projection: the value of a token is its key AS PROJECTED
  (before norm and rotation);
* ``positions``: a ``rotary_partial`` part (the first ``dims`` entries of a head rotate) or None;
* ``softcap``: score <- softcap * tanh(score / softcap) after the scale; None: off;
* ``window``: a query at position i sees the keys j with 0 <= i - j < window; None: all before it;
* ``chunk``: a query at position i sees the keys j <= i of its own chunk, floor(j / chunk) = floor(i / chunk), chunks
  counted from position 0 of the sequence (not together with ``window``);
* ``v_dim``: the value size of a head where it differs from the key size (default ``head_dim``);
* ``sink``: one is added to the softmax's denominator, p_j = exp(s_j) / (1 + sum exp(s_j)); "learned": exp(sink_h) is,
  one number a query head (tensor ``sink`` [H]), not scaled;
* ``gate`` "sigmoid": the concatenated heads are multiplied by sigmoid(W_g x) before the output
  projection; "head_sigmoid": W_g has one row a head, whose number multiplies the whole head; None: no gate;
* ``value_rotation``: a ``rotary_partial`` part over the value heads: the value of position j turns by j before it is
  cached, and every head's output at position i turns back by i, so a value counts by its distance; None: values stay;
* ``bias``: q, k and v have biases (tensors ``q.b``, ``k.b``, ``v.b``), added before the norm;
* ``keep_first``: with a ``window``, the sequence's first that many tokens stay visible to every later query, at their
  true positions (their pages are never given back);
* ``score_mix``: the scaled scores of the heads are mixed before the softmax, s_h <- sum_g talk[h, g] s_g (tensor ``talk``
  [H, H]);
* ``value_mix``: "first": this layer's values of the step's tokens are left to later layers; "later": before they are
  cached, v <- (1 - l) v + l v_first, with those values and l = ``vmix`` (a tensor of one number); None: neither.

Query head h reads KV head h // (heads / kv_heads).  The input products (q, k, the gate) run as ONE
product with float32 output, because norm and rotation are float32; one kernel then norms, rotates
and writes q and the cache rows (csrc/gated_attention.cu), and the paged attention kernels of the
plain attention mixer do the rest with softcap, sink and gate as arguments.  With any of the last four options the kernel
between product and attention is csrc/qkv_prepare.cu, which also takes over split sums the product left (few tokens) and
pads key and value rows of different sizes itself; the attention kernels are chosen by parts/mixed_attention_bf16.py
(bfloat16) or are the one-warp-a-row kernel.  Mixed scores are linear in the queries, so that kernel spreads each mixed
query over all KV heads (see there), and a head's score is one dot product over all of a token's keys.

Without those options, heads whose key and value sizes differ are laid out at load time in rows of one padded size P (the larger of the two,
rounded up to a multiple of 8): zero rows in W_q, W_k and W_v, zero columns in W_o, so that scores and outputs are what they were and every paged
kernel sees heads of P entries.  A position part with ``pairing`` "interleaved" has the rows of W_q and W_k laid out
by its ``permutation()`` in the same pass.

Parameters: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim``, ``scale``, ``eps`` and the
options above.  Tensors below the prefix: q [H D, hidden], k [G D, hidden], (v [G V, hidden]),
q.norm [H D], k.norm [G D], g [H V or H, hidden], sink [H], talk [H, H], vmix [], o [hidden, H V].
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..config.spec import PartSpec
from .base import MIXERS, POSITIONS, KVSpec, Mixer, TensorSpec, build_part
from .linear import Linear


@MIXERS.register("gated_attention")
class GatedAttentionMixer(Mixer):
    graph_safe = True  # nothing is planned on the host for single-token steps

    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.num_heads = int(p["num_heads"])
        self.num_kv_heads = int(p["num_kv_heads"])
        self.qk_dim = int(p["head_dim"])
        self.v_dim = int(p["v_dim"]) if p.get("v_dim") is not None else self.qk_dim
        # the size of a head as the kernels and the pages see it: the larger of the two where they differ (then rounded up
        # to a multiple of 8, which the kernels' 16-byte loads want)
        self.head_dim = self.qk_dim if self.v_dim == self.qk_dim else -(-max(self.qk_dim, self.v_dim) // 8) * 8
        self.bias = bool(p.get("bias", False))
        self.score_mix = bool(p.get("score_mix", False))
        self.value_mix = p.get("value_mix")
        self.keep_first = int(p.get("keep_first", 0) or 0) if p.get("window") else 0
        # whether csrc/qkv_prepare.cu stands between product and attention (it pads rows itself, to a size the tensor-core
        # kernels take where there is one)
        self.prepared = self.bias or self.score_mix or self.value_mix is not None or self.keep_first > 0
        if self.prepared:
            size = max(self.qk_dim, self.v_dim)
            self.head_dim = 64 if size <= 64 else (128 if size <= 128 else -(-size // 8) * 8)
        self.padded = self.head_dim != self.qk_dim or self.head_dim != self.v_dim
        self.scale = float(p["scale"]) if p.get("scale") is not None else self.qk_dim ** -0.5
        self.softcap: Optional[float] = float(p["softcap"]) if p.get("softcap") else None
        self.chunk: Optional[int] = int(p["chunk"]) if p.get("chunk") else None
        if self.chunk is not None and p.get("window"):
            raise ValueError("a window and a chunked mask do not go together")
        # the mask code of the paged kernels: positive a sliding window, negative the chunk size, None neither
        self.window: Optional[int] = -self.chunk if self.chunk is not None else (int(p["window"]) if p.get("window") else None)
        self.learned_sink = p.get("sink") == "learned"
        self.sink = bool(p.get("sink", False))  # with "learned": the heads' scores, a tensor, from ``load`` on
        self.values_from_keys = bool(p.get("values_from_keys", False))
        self.qk_norm = p.get("qk_norm")
        self.gate = p.get("gate")
        self.eps = float(p.get("eps", 1e-6))
        if self.qk_norm not in (None, "whole"):
            raise ValueError(f"unknown qk_norm {self.qk_norm!r} (known: 'whole', None)")
        if self.gate not in (None, "sigmoid", "head_sigmoid"):
            raise ValueError(f"unknown gate {self.gate!r} (known: 'sigmoid', 'head_sigmoid', None)")
        if p.get("sink", False) not in (False, True, None, "learned"):
            raise ValueError(f"unknown sink {p['sink']!r} (known: True, False, 'learned')")
        if self.num_heads % self.num_kv_heads:
            raise ValueError("num_heads must be divisible by num_kv_heads")
        if self.head_dim > 256:
            raise ValueError(f"head_dim {self.head_dim} is not supported (up to 256)")
        if self.value_mix not in (None, "first", "later"):
            raise ValueError(f"unknown value_mix {self.value_mix!r} (known: 'first', 'later', None)")
        if self.prepared and (p.get("softcap") or p.get("chunk") or p.get("sink") or self.gate or self.values_from_keys
                              or p.get("value_rotation")):
            raise ValueError("biases, mixed scores, mixed values and kept first tokens are not built together with a score "
                             "cap, a chunked mask, a sink, a gate, values taken from the keys or rotated values")
        if not self.prepared and self.padded and (self.qk_norm is not None or self.values_from_keys):
            raise ValueError("heads whose key and value sizes differ are not built together with a norm over the whole "
                             "projection or with values taken from the keys")
        self.positions = build_part(POSITIONS, p["positions"]) if p.get("positions") else None
        if self.positions is not None and not hasattr(self.positions, "inv_freq"):
            raise ValueError("this mixer rotates inside its own kernel and needs a position part with a frequency table")
        self.value_rotation = build_part(POSITIONS, p["value_rotation"]) if p.get("value_rotation") else None
        if self.value_rotation is not None and (
                not hasattr(self.value_rotation, "inv_freq") or self.value_rotation.head_dim != self.v_dim
                or getattr(self.value_rotation, "scaling", None) or self.values_from_keys):
            raise ValueError("the values' rotation is a position part with a frequency table over the value size, without "
                             "frequency scaling, for values with a projection of their own")
        self.q_size = self.num_heads * self.head_dim
        self.kv_size = self.num_kv_heads * self.head_dim
        self.in_proj: Linear | None = None
        self.o_proj: Linear | None = None
        self.q_norm = self.k_norm = None
        self.talk = self.value_lambda = None

    def kv_spec(self) -> KVSpec:
        # a chunk's keys all lie within ``chunk`` positions of the query: pages are given back as for a window of that size
        return KVSpec(self.num_kv_heads, self.head_dim, self.chunk if self.chunk is not None else self.window,
                      keep_first=self.keep_first)

    @classmethod
    def expected_tensors(cls, spec: PartSpec, prefix: str) -> list[TensorSpec]:
        p = spec.params
        hidden, d = int(p["hidden_size"]), int(p["head_dim"])
        dv = int(p["v_dim"]) if p.get("v_dim") is not None else d
        q_size, kv_size = int(p["num_heads"]) * d, int(p["num_kv_heads"]) * d
        out = [TensorSpec(prefix + "q", (q_size, hidden)), TensorSpec(prefix + "k", (kv_size, hidden))]
        if not p.get("values_from_keys", False):
            out.append(TensorSpec(prefix + "v", (int(p["num_kv_heads"]) * dv, hidden)))
        if p.get("bias", False):
            out += [TensorSpec(t.name + ".b", (t.shape[0],), init="zeros") for t in list(out)]
        if p.get("score_mix", False):
            out.append(TensorSpec(prefix + "talk", (int(p["num_heads"]), int(p["num_heads"])), init="eye"))
        if "value_mix" in p:  # a layer of such a design without value mixing may carry the number all the same; nothing reads it
            out.append(TensorSpec(prefix + "vmix", (), init="zeros", optional=p["value_mix"] is None))
        if p.get("qk_norm") == "whole":
            out += [TensorSpec(prefix + "q.norm", (q_size,), init="ones"), TensorSpec(prefix + "k.norm", (kv_size,), init="ones")]
        if p.get("gate") == "sigmoid":
            out.append(TensorSpec(prefix + "g", (int(p["num_heads"]) * dv, hidden)))
        if p.get("gate") == "head_sigmoid":
            out.append(TensorSpec(prefix + "g", (int(p["num_heads"]), hidden)))
        if p.get("sink") == "learned":
            out.append(TensorSpec(prefix + "sink", (int(p["num_heads"]),), init="zeros"))
        out.append(TensorSpec(prefix + "o", (hidden, int(p["num_heads"]) * dv)))
        if p.get("positions"):
            out += POSITIONS.get(p["positions"].kind).expected_tensors(p["positions"], prefix)
        return out

    def _load_prepared(self, tensors: dict, prefix: str, device, dtype) -> None:
        """The projections as the checkpoint has them (unpadded), in the order [q; k; v], every q and k head's rows, biases
        and norm weights in the order in which the kernels' split-half rotation turns the checkpoint's pairs."""
        D, order = self.qk_dim, self.positions.permutation() if self.positions is not None else None

        def ordered(name: str, suffix: str = "") -> torch.Tensor:
            w = tensors[prefix + name + suffix]
            if name == "v" or order is None:
                return w
            return w.reshape(-1, D, *w.shape[1:])[:, order].reshape(w.shape)

        names = ("q", "k", "v")
        rows = [ordered(n) for n in names]
        biases = [ordered(n, ".b").float() for n in names] if self.bias else []
        odd = -sum(w.shape[0] for w in rows) % 4
        if odd:  # zero rows behind the last: float32 output rows of whole 16-byte pieces
            rows.append(rows[-1].new_zeros(odd, rows[-1].shape[1]))
            if biases:
                biases.append(biases[-1].new_zeros(odd))
        self.in_proj = Linear(torch.cat(rows, dim=0), torch.cat(biases) if biases else None, device, dtype)
        self.o_proj = Linear(tensors[prefix + "o"], None, device, dtype)
        f32 = lambda w: w.to(device=device, dtype=torch.float32).contiguous()
        if self.qk_norm == "whole":
            self.q_norm, self.k_norm = f32(ordered("q", ".norm")), f32(ordered("k", ".norm"))
        if self.score_mix:
            self.talk = f32(tensors[prefix + "talk"])
        if self.value_mix == "later":
            self.value_lambda = f32(tensors[prefix + "vmix"]).reshape(1)
        if self.positions is not None:
            self.positions.load(tensors, prefix, device, dtype)
        self.proj_size = self.in_proj.out_features

    def load(self, tensors: dict, prefix: str, device, dtype) -> None:
        if self.prepared:
            self._load_prepared(tensors, prefix, device, dtype)
            return
        names = ["q", "k"] + ([] if self.values_from_keys else ["v"]) + (["g"] if self.gate else [])
        part = self.value_rotation
        v_order = part.permutation() if part is not None and hasattr(part, "permutation") else None
        order = self.positions.permutation() if self.positions is not None and hasattr(self.positions, "permutation") else None
        P = self.head_dim

        def heads_of(name: str, size: int, order) -> torch.Tensor:
            """The projection ``name`` with every head's ``size`` rows in the kernels' order, padded to P rows."""
            w = tensors[prefix + name]
            if size == 1 and name == "g":  # one row a head
                return w
            if not self.padded and (order is None or order == list(range(size))):
                return w
            w = w.reshape(-1, size, w.shape[1])
            if order is not None:
                w = w[:, order]
            if size != P:
                w = torch.cat([w, w.new_zeros(w.shape[0], P - size, w.shape[2])], dim=1)
            return w.reshape(-1, w.shape[2])

        sizes = {"q": (self.qk_dim, order), "k": (self.qk_dim, order), "v": (self.v_dim, v_order),
                 "g": (1, None) if self.gate == "head_sigmoid" else (self.v_dim, v_order)}
        rows = [heads_of(n, *sizes[n]) for n in names]
        odd = -sum(w.shape[0] for w in rows) % 4
        if odd:  # zero rows behind the last: float32 output rows of whole 16-byte pieces
            rows.append(rows[-1].new_zeros(odd, rows[-1].shape[1]))
        self.in_proj = Linear(torch.cat(rows, dim=0), None, device, dtype)
        w_o = tensors[prefix + "o"]
        if v_order is not None and v_order != list(range(self.v_dim)):  # the heads' outputs come in the values' order
            w_o = w_o.reshape(w_o.shape[0], self.num_heads, self.v_dim)[:, :, v_order].reshape(w_o.shape[0], -1)
        if self.padded:  # zero columns where the heads' outputs are padded
            w_o = w_o.reshape(w_o.shape[0], self.num_heads, self.v_dim)
            w_o = torch.cat([w_o, w_o.new_zeros(w_o.shape[0], self.num_heads, P - self.v_dim)], dim=2).reshape(w_o.shape[0], -1)
        self.o_proj = Linear(w_o, None, device, dtype)
        if self.qk_norm == "whole":
            self.q_norm = tensors[prefix + "q.norm"].to(device=device, dtype=torch.float32).contiguous()
            self.k_norm = tensors[prefix + "k.norm"].to(device=device, dtype=torch.float32).contiguous()
        if self.positions is not None:
            self.positions.load(tensors, prefix, device, dtype)
        if self.value_rotation is not None:
            self.value_rotation.load(tensors, prefix, device, dtype)
        if self.learned_sink:
            self.sink = tensors[prefix + "sink"].to(device=device, dtype=torch.float32).contiguous()
        # where the projection rows hold the values and the gate
        self.v_offset = self.q_size if self.values_from_keys else self.q_size + self.kv_size
        self.gate_offset = self.q_size + self.kv_size * (1 if self.values_from_keys else 2)
        self.proj_size = self.in_proj.out_features

    def _forward_prepared(self, ctx, x, acc, cache) -> None:
        from . import mixed_attention_bf16

        tokens, H, G = x.shape[0], self.num_heads, self.num_kv_heads
        sums = self.in_proj.deferred(ctx, x)
        if sums is not None:  # few tokens: the product's split sums are completed by the kernel behind it
            source = {"src": sums[0], "splits": sums[1], "row": self.proj_size, "bias": self.in_proj.bias}
        else:
            proj = ctx.buffer("gated_attention.proj", (tokens, self.proj_size), torch.float32)
            self.in_proj.forward(x, proj)
            source = {"src": proj}
        v_first = None
        if self.value_mix is not None:
            v_first = ctx.buffer("gated_attention.first_values", (tokens, G * self.v_dim), torch.float32)
        # how the attention kernels want the queries of mixed scores: spread over all KV heads, or as they are for the
        # kernels that mix the scores themselves
        spread = mixed_attention_bf16.query_form(self, ctx, cache) if self.score_mix else 0
        span = G if spread else 1
        q = ctx.buffer("gated_attention.spread_q" if spread else "gated_attention.q", (tokens, H * span * self.head_dim), ctx.dtype)
        positions = self.positions
        ops.qkv_prepare(
            sizes=(H, G, self.qk_dim, self.v_dim, self.head_dim), positions=ctx.positions, token_req=ctx.token_req,
            req_indptr=ctx.req_indptr, block_table=cache.block_table, pages=cache.pages, page_size=cache.page_size, q_out=q,
            wq=self.q_norm, wk=self.k_norm, eps=self.eps, inv_freq=positions.inv_freq if positions is not None else None,
            magnitude=positions.magnitude if positions is not None else 1.0, mix=self.talk, spread=spread, v_first=v_first,
            value_lambda=self.value_lambda, write_kv=cache.writable, **source)
        out = ctx.buffer("gated_attention.out", (tokens, H * self.v_dim), ctx.dtype)
        if not mixed_attention_bf16.forward(self, ctx, q, cache, out):
            ops.attention_generic(q, q.stride(0), cache.pages, cache.block_table, ctx.token_req, ctx.positions, out, tokens,
                                  H, G, self.head_dim, cache.page_size, self.window, self.scale, keep=self.keep_first,
                                  spread=bool(spread), v_cols=self.v_dim)
        if not self.o_proj.accumulate_later(ctx, out, acc):
            self.o_proj.forward(out, acc, accumulate=True)

    def forward(self, ctx, x, acc, cache) -> None:
        if self.prepared:
            self._forward_prepared(ctx, x, acc, cache)
            return
        tokens = x.shape[0]
        proj = ctx.buffer("gated_attention.proj", (tokens, self.proj_size), torch.float32)
        self.in_proj.forward(x, proj)
        q = ctx.buffer("gated_attention.q", (tokens, self.q_size), ctx.dtype)
        positions = self.positions
        ops.normed_qk_store(
            proj, self.q_norm, self.k_norm, positions.inv_freq if positions is not None else None,
            positions.magnitude if positions is not None else 1.0, self.eps, ctx.positions, ctx.token_req,
            cache.block_table, cache.pages, cache.page_size, q, self.num_heads, self.num_kv_heads, self.head_dim,
            positions.dims if positions is not None else 0, self.v_offset, write_kv=cache.writable,
            v_inv_freq=self.value_rotation.inv_freq if self.value_rotation is not None else None)
        out = ctx.buffer("gated_attention.out", (tokens, self.q_size), ctx.dtype)
        gate = proj[:, self.gate_offset:] if self.gate == "sigmoid" else None
        if gate is not None and self.value_rotation is not None:
            gate = None  # the output turns back first: the gate follows behind the attention kernel
        from . import attention_bf16

        # bfloat16 heads of 64 or 128: the tensor-core kernel (tiles of 16 packed rows for single tokens, of 64
        # for prompt portions); else, and in float32, one warp per (token, head)
        if not (ctx.dtype == torch.bfloat16 and attention_bf16.forward(self, ctx, q, cache, out, gate=gate)):
            ops.attention_generic(q, q.stride(0), cache.pages, cache.block_table, ctx.token_req, ctx.positions, out, tokens,
                                  self.num_heads, self.num_kv_heads, self.head_dim, cache.page_size, self.window, self.scale,
                                  softcap=self.softcap, sink=self.sink, gate=gate)
        if self.value_rotation is not None or self.gate == "head_sigmoid":
            ops.head_finish(out, ctx.positions, self.value_rotation.inv_freq if self.value_rotation is not None else None,
                            proj[:, self.gate_offset:] if self.gate == "head_sigmoid" else None, self.num_heads, self.head_dim)
        if self.value_rotation is not None and self.gate == "sigmoid":
            ops.gate_mul_(out, proj[:, self.gate_offset:self.gate_offset + self.q_size])
        if not self.o_proj.accumulate_later(ctx, out, acc):
            self.o_proj.forward(out, acc, accumulate=True)
