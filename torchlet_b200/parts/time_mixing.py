"""Time mixing with a data-dependent decay and a bonus for the current token: a recurrent mixer with one D x D float32
state matrix per head and request (key channel x value channel) and the request's last input row, both kept in the
request's slot between steps.

With x' the row of the token before (zeros before the first), each of r, k, v, g and w reads its own mix
m_c = x + (x' - x) * mu_c (csrc/token_shift.cu); r = W_r m_r, k = W_k m_k, v = W_v m_v (heads x D),
gate = silu(W_g m_g), and a decay per key channel a = exp(-exp(W_w2 tanh(W_w1 m_w) + w0)).  Per head:

    o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t        S_t = diag(a_t) S_(t-1) + k_t v_t^T

Each head's o is divided by its root mean square; the heads, concatenated, are multiplied by a weight over all of them
and by the gate, and go through W_o into the stream.  The products r, k, v and g run over the mixes' planes and leave
float32 planes, which the scan of the gated linear attention reads (csrc/gla.cu); decay, state, recurrence and norm are
float32 in both engines.  A step of single tokens in bfloat16 runs all five products as one launch over the stacked
matrices and everything from their split sums to the gated heads as one kernel (csrc/time_mixing.cu).

Parameters: ``hidden_size``, ``num_heads``, ``head_dim``, ``decay_rank``, ``eps``.  Tensors below the prefix: r, k, v, g
[H D, hidden]; w1 [rank, hidden]; w2 [H D, rank]; w0, norm [H D]; u [H, D]; mu.r, mu.k, mu.v, mu.g, mu.w [hidden];
o [hidden, H D].
"""
from __future__ import annotations

import torch

from .. import ops
from ..config.spec import PartSpec
from .base import MIXERS, Mixer, StateSpec, TensorSpec
from .linear import Linear

PRODUCTS = ("r", "k", "v", "g")  # the order of the planes
MIXES = PRODUCTS + ("w",)


@MIXERS.register("time_mixing")
class TimeMixing(Mixer):
    graph_safe = True  # nothing is planned on the host: requests and slots are read on the device

    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.num_heads = int(p["num_heads"])
        self.head_dim = int(p["head_dim"])
        self.rank = int(p["decay_rank"])
        self.eps = float(p["eps"])
        if self.head_dim > 256:
            raise ValueError(f"head_dim {self.head_dim} is not supported by the scan kernel (up to 256)")
        if self.rank > 1024:
            raise ValueError(f"a decay rank of {self.rank} is not supported (up to 1024)")
        self.size = self.num_heads * self.head_dim
        self.stacked = None  # [4 H D + rank, hidden]: the five input matrices; the products below are views of it
        self.products: list = []
        self.w1_proj: Linear | None = None
        self.o_proj: Linear | None = None
        self.mu = self.w2 = self.w0 = self.bonus = self.norm_weight = None

    def state_spec(self) -> dict:
        return {"shift": StateSpec((self.hidden_size,), "float32"),
                "matrix": StateSpec((self.num_heads, self.head_dim, self.head_dim), "float32")}

    @classmethod
    def expected_tensors(cls, spec: PartSpec, prefix: str) -> list[TensorSpec]:
        p = spec.params
        hidden, rank, H, D = int(p["hidden_size"]), int(p["decay_rank"]), int(p["num_heads"]), int(p["head_dim"])
        out = [TensorSpec(f"{prefix}mu.{c}", (hidden,)) for c in MIXES]
        out += [TensorSpec(prefix + c, (H * D, hidden)) for c in PRODUCTS]
        out += [TensorSpec(prefix + "w1", (rank, hidden)), TensorSpec(prefix + "w2", (H * D, rank)),
                TensorSpec(prefix + "w0", (H * D,)), TensorSpec(prefix + "u", (H, D)),
                TensorSpec(prefix + "norm", (H * D,), init="ones"), TensorSpec(prefix + "o", (hidden, H * D))]
        return out

    def load(self, tensors: dict, prefix: str, device, dtype) -> None:
        self.stacked = torch.cat([tensors[prefix + c] for c in PRODUCTS] + [tensors[prefix + "w1"]]).to(
            device=device, dtype=dtype).contiguous()
        self.products = [Linear.from_device_weight(self.stacked[i * self.size:(i + 1) * self.size]) for i in range(len(PRODUCTS))]
        self.w1_proj = Linear.from_device_weight(self.stacked[len(PRODUCTS) * self.size:])
        self.one_kernel = (dtype == torch.bfloat16 and self.hidden_size % 8 == 0
                           and ops.time_mixing_step_supported(self.num_heads, self.head_dim, self.rank))
        self.o_proj = Linear(tensors[prefix + "o"], None, device, dtype)
        f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
        self.mu = f32(torch.stack([tensors[f"{prefix}mu.{c}"] for c in MIXES]))
        self.w0, self.bonus, self.norm_weight = (f32(tensors[prefix + n]) for n in ("w0", "u", "norm"))
        self.w2 = f32(tensors[prefix + "w2"]).t().contiguous()  # [rank, H D]: threads of a block read consecutive entries

    def forward(self, ctx, x, acc, cache) -> None:
        tokens, H, D = x.shape[0], self.num_heads, self.head_dim
        # scratch sized once for the largest step: its addresses never change
        capacity = max(ctx.token_capacity, tokens, ops.STACKED_ROWS[-1])

        def planes_of(name: str, count: int, width: int, dtype, rows: int = tokens):
            return ctx.buffer(name, (count * capacity, width), dtype)[:count * rows].view(count, rows, width)

        out = ctx.buffer("time_mixing.out", (tokens, self.size), ctx.dtype)
        if self.one_kernel and ctx.decode_only and tokens <= ops.STACKED_ROWS[-1]:
            rows = next(n for n in ops.STACKED_ROWS if tokens <= n)
            mixes = planes_of("time_mixing.mixes", len(MIXES), self.hidden_size, ctx.dtype, rows)
            ops.token_shift(x, self.mu, mixes, cache.state["shift"], ctx.token_req, ctx.req_indptr, ctx.slots, ctx.num_requests)
            sums, splits = ops.gemm_tc_stacked(mixes, self.stacked, self.size)
            ops.time_mixing_step(sums, splits, rows, self.w2, self.w0, self.bonus, self.norm_weight, ctx.slots,
                                 cache.state["matrix"], out, H, D, self.eps)
            if not self.o_proj.accumulate_later(ctx, out, acc):
                self.o_proj.forward(out, acc, accumulate=True)
            return
        mixes = planes_of("time_mixing.mixes", len(MIXES), self.hidden_size, ctx.dtype)
        ops.token_shift(x, self.mu, mixes, cache.state["shift"], ctx.token_req, ctx.req_indptr, ctx.slots, ctx.num_requests)
        planes = planes_of("time_mixing.planes", len(PRODUCTS), self.size, torch.float32)
        for product, mix, plane in zip(self.products, mixes, planes):
            product.forward(mix, plane)
        low = ctx.buffer("time_mixing.low", (tokens, self.rank), torch.float32)
        self.w1_proj.forward(mixes[-1], low)
        decay = ctx.buffer("time_mixing.decay", (tokens, self.size), torch.float32)
        ops.gla_decay(low, 0, self.w2, self.w0, decay, self.rank, 0.0)
        o = ctx.buffer("time_mixing.o", (tokens, self.size), torch.float32)
        plane = tokens * self.size
        ops.gla_scan(planes[0], decay, ctx.req_indptr, ctx.slots, cache.state["matrix"], o, ctx.num_requests, H, D, D, 1.0,
                     bonus=self.bonus, k_offset=plane, v_offset=2 * plane)
        ops.gla_finish(o, planes[3], 0, self.norm_weight, out, H, D, self.eps)
        if not self.o_proj.accumulate_later(ctx, out, acc):
            self.o_proj.forward(out, acc, accumulate=True)
