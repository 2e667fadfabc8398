"""Small Lidizen configurations of the tests, their random weights, and an engine around them.  No two agree in any size:
one stream and several, one KV head and as many as heads, key and value sizes that differ either way and are no multiple of
8, windows of one token, shorter than a page and of several pages, no kept token, one, more than a page and more than the
window, a rotation over all entries and over a few, layers with and without value mixing (the first layer among them), a
layer without a feed-forward, one expert of one, every expert of three, a table of one pair row, scales that are no power
of the key size."""
from __future__ import annotations

import copy
import functools

import torch

import plain_lidizen
from fusolix_cases import replay  # noqa: F401  (one request in portions, every position's logits)

# Largest allowed |engine - plain| of a position's logits as a fraction of that position's largest |logit|.
TOLERANCE = {"float32": 1e-4, "bfloat16": 6e-2}


def mixer(heads, kv_heads, dim, vdim, scale, size, keep, rot_dims, base=10000.0, v_mix=True):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix,
            "mask": {"size": size, "keep_first": keep}, "rot": {"base": base, "dims": rot_dims}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(m, mlp):
    return {"type": "attention", "mixer": m, "mlp": mlp}


def config(vocab, width, streams, eps, pairs, *layers):
    return {"architecture": "Lidizen", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), pairs))}, "layers": list(layers)}


CASES = {
    # three streams; windows shorter than a page and of several; kept tokens: fewer than a page, one, more than the window,
    # none; values mixed from the second layer on, one layer between without
    "P": config(101, 96, 3, 1e-5, (37, 5, 3),
                layer(mixer(4, 2, 24, 16, 0.21, 13, 5, 24, v_mix=False), dense(40)),
                layer(mixer(4, 2, 20, 12, 0.3, 37, 1, 8, 500.0), moe(6, 2, 24)),
                layer(mixer(6, 3, 16, 12, 0.25, 7, 18, 16, v_mix=False), None),
                layer(mixer(2, 2, 12, 12, 0.28, 20, 0, 6, 500.0), moe(3, 3, 56))),
    # one stream, one head, a window of ONE token, more kept tokens than a page, one pair row, one expert of one; odd sizes
    "Q": config(67, 44, 1, 1e-6, (1, 3, 11),
                layer(mixer(1, 1, 10, 18, 0.4, 1, 3, 10, 100.0), moe(1, 1, 20)),
                layer(mixer(5, 1, 18, 18, 0.2, 9, 21, 2, 100.0, v_mix=False), dense(36)),
                layer(mixer(3, 1, 14, 18, 0.33, 30, 30, 14, 100.0), moe(5, 1, 12))),
    # head sizes of 64 and 128 (the tensor-core kernels without padding), groups of 1, 2, 4 and 9 heads, windows and kept
    # tokens over several pages and key tiles
    "R": config(211, 128, 4, 1e-6, (500, 31, 17),
                layer(mixer(8, 2, 64, 64, 0.11, 150, 40, 64, 50000.0, v_mix=False), moe(8, 2, 64)),
                layer(mixer(4, 4, 128, 64, 0.09, 70, 20, 32, 50000.0), dense(192)),
                layer(mixer(8, 4, 64, 64, 0.1, 33, 140, 64, 50000.0), None),
                layer(mixer(9, 1, 64, 128, 0.12, 40, 8, 16, 50000.0, v_mix=False), dense(64))),
    # no mask at all in one layer, no rotation in another, no value mixing anywhere, two streams, no pair table
    "S": {"architecture": "Lidizen", "vocab": 53, "width": 48, "streams": 2, "norm": {"eps": 1e-5},
          "layers": [layer({"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.25, "rot": {"base": 1000.0, "dims": 4}},
                           moe(4, 2, 32)),
                     layer({"heads": 3, "kv_heads": 3, "dim": 8, "vdim": 16, "scale": 0.35,
                            "mask": {"size": 5, "keep_first": 2}}, dense(64))]},
    # head sizes the tensor-core attention does not take, five streams, more than 16 heads a KV head
    "T": config(61, 56, 5, 1e-5, (211, 2, 9),
                layer(mixer(2, 1, 136, 24, 0.1, 11, 4, 40), dense(24)),
                layer(mixer(17, 1, 8, 24, 0.4, 19, 9, 8), moe(4, 3, 16))),
}


def _all_experts(case: dict) -> dict:
    case = copy.deepcopy(case)
    for entry in case["layers"]:
        if entry["mlp"] is not None and entry["mlp"]["kind"] == "moe":
            entry["mlp"]["router"]["top"] = entry["mlp"]["router"]["experts"]
    return case


# "Pa", ..: the same models with EVERY expert chosen.  Random routers have close calls: where two experts' logits lie within
# bfloat16 rounding of one another the bfloat16 engine may choose the other one, and that position, and through keys all
# behind it, then differs by a whole expert's output.  So the bfloat16 engine is compared on these (same tensors, no discrete
# choice), the float32 engine on the true routing; the choice itself is tested on given inputs.
CASES.update({name + "a": _all_experts(case) for name, case in list(CASES.items())})


def variant(name: str, dtype: str) -> str:
    return name if dtype == "float32" else name + "a"


def config_for(name: str):
    from torchlet_b200.config import LidizenConfig

    return LidizenConfig.from_dict(CASES[name])


@functools.lru_cache(maxsize=None)
def weights_for(name: str, seed: int = 0):
    """bfloat16-rounded random weights as float32 tensors by name (so that both engines and the plain implementation hold
    the same numbers).  Routers are drawn wider; mixing matrices, the streams' vectors, biases and the value-mixing numbers
    are drawn away from the identity, one and zero, so that each counts."""
    from torchlet_b200.weights import random_tensors

    tensors = random_tensors(config_for(name), seed=700 + seed, std=0.1, norm_std=0.1, dtype="bfloat16")
    g = torch.Generator().manual_seed(1100 + seed)
    out = {}
    for k, v in tensors.items():
        v = v.float()
        noise = torch.randn(v.shape, generator=g)
        if k.endswith(".router"):
            v = v * 4
        elif ".hc" in k:
            v = v + 0.3 * noise
        elif k.endswith(".talk"):
            v = v + 0.4 * noise
        elif k.endswith(".vmix"):
            v = 0.35 + 0.1 * noise
        elif k.endswith(".b"):
            v = 0.2 * noise
        elif k in ("embed", "bigram"):
            v = v * 5
        out[k] = v.to(torch.bfloat16).float()
    return out


def make_ids(name: str, length: int, seed: int):
    g = torch.Generator().manual_seed(5000 + seed)
    return torch.randint(0, CASES[name]["vocab"], (length,), generator=g).tolist()


@functools.lru_cache(maxsize=None)
def plain_logits(name: str, length: int, seed: int):
    ids = make_ids(name, length, seed)
    return ids, plain_lidizen.forward(weights_for(name), CASES[name], ids).float()


def make_model(name: str, dtype: str, weights=None):
    from torchlet_b200.engine.loading import build_model

    w = weights if weights is not None else weights_for(name)
    return build_model(config_for(name), {k: v.to(torch.bfloat16) for k, v in w.items()}, dtype)


def make_runner(name: str, dtype: str, num_pages: int = 64, slots: int = 4, page_size: int = 16, budget: int = 512,
                max_seq_len: int = 512, cuda_graph: bool = False, weights=None):
    from torchlet_b200.config import EngineConfig
    from torchlet_b200.engine import ModelRunner

    engine = EngineConfig(dtype=dtype, max_decode_slots=slots, kv_block_size=page_size, max_num_blocks=num_pages,
                          max_seq_len=max_seq_len, max_num_batched_tokens=budget, cuda_graph=cuda_graph)
    return ModelRunner(make_model(name, dtype, weights), engine)


def assert_close(got, want, dtype: str, what: str = ""):
    """Row by row: the largest difference of a position's logits against the largest |logit| of that position."""
    assert got.shape == want.shape, f"{what}: shapes {tuple(got.shape)} and {tuple(want.shape)}"
    assert torch.isfinite(got).all(), f"{what}: not finite"
    got, want = got.reshape(-1, got.shape[-1]).double(), want.reshape(-1, want.shape[-1]).double()
    err, scale = (got - want).abs().amax(dim=1), want.abs().amax(dim=1)
    worst = int((err / scale).argmax())
    assert err[worst] <= TOLERANCE[dtype] * scale[worst], (
        f"{what}: row {worst}: max |diff| {err[worst]:.3e} > {TOLERANCE[dtype]:.1e} * {scale[worst]:.3f}")
