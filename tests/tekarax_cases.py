"""Small Tekarax configurations of the tests, their random weights, and an engine around them.  No two agree in any
size: key and value sizes that differ and are no multiple of 8, one head and several, one key/value head and as many as
query heads, windows of one token, of less than a page, of several pages and longer than every test sequence, a rotation
over all entries and over a few, frequencies slowed down or not, decay ranks from one up, routers of one expert and of
several with and without a shared expert, a layer without a feed-forward, a looped stretch at the start, in the middle,
at the end, run once and several times, and no loop."""
from __future__ import annotations

import copy
import functools

import torch

import plain_tekarax

# Largest allowed |engine - plain| of a position's logits as a fraction of that position's largest |logit|.
TOLERANCE = {"float32": 1e-4, "bfloat16": 6e-2}


def rot(base, dims, scaling=None):
    out = {"base": base, "dims": dims}
    if scaling is not None:
        out["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return out


def attention(heads, kv_heads, dim, vdim, scale, rotation, mlp):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rotation}}


def latent(heads, dim, vdim, kv_rank, scale, size, mlp):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "mask": {"size": size}}}


def wkv(heads, dim, rank, mlp):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "decay_rank": rank}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


CASES = {
    # a looped stretch in the middle, three times; windows of 13 and 5 tokens (less than a page, no power of two); a
    # rotation over 8 of 24 entries with slowed frequencies; a layer without a feed-forward
    "P": {"architecture": "Tekarax", "vocab": 101, "width": 96, "norm": {"eps": 1e-5},
          "loop": {"start": 1, "stop": 3, "times": 3},
          "layers": [
              wkv(3, 12, 7, moe(6, 2, 24, shared=40)),
              attention(4, 2, 24, 16, 0.3, rot(500.0, 8, (8.0, 1.0, 4.0, 64)), dense(40)),
              latent(3, 20, 28, 40, 0.2, 13, moe(5, 3, 24)),
              latent(2, 8, 12, 24, 0.5, 5, None),
              wkv(2, 24, 16, None),
          ]},
    # ones: one head everywhere, a window of ONE token, a decay rank of one, one expert, every expert of three, the loop
    # at the very end and run ONCE, frequencies as they are
    "Q": {"architecture": "Tekarax", "vocab": 67, "width": 64, "norm": {"eps": 1e-6},
          "loop": {"start": 1, "stop": 3, "times": 1},
          "layers": [
              latent(1, 8, 8, 16, 0.35, 1, moe(1, 1, 24, shared=16)),
              attention(1, 1, 40, 8, 0.2, rot(10000.0, 40), moe(3, 3, 24)),
              wkv(1, 8, 1, dense(72)),
          ]},
    # sizes the tensor-core kernels take: attention heads of 64 and 128, windows over several pages and key tiles, a
    # time mixing of 64 x 64, experts of 64; no loop
    "R": {"architecture": "Tekarax", "vocab": 211, "width": 128, "norm": {"eps": 1e-6},
          "layers": [
              attention(4, 1, 64, 64, 0.125, rot(50000.0, 32, (4.0, 1.0, 2.0, 32)), moe(8, 2, 64, shared=64)),
              latent(4, 32, 32, 64, 0.125, 48, dense(192)),
              wkv(2, 64, 24, moe(4, 2, 64)),
              attention(4, 2, 128, 128, 0.09, rot(50000.0, 128), dense(96)),
              latent(6, 64, 48, 96, 0.1, 150, None),
          ]},
    # sizes that are no multiple of 8 (the products' and the attention's any-size kernels in both engines), a window
    # longer than every test sequence, as many key/value heads as heads, the loop at the very start, twice
    "S": {"architecture": "Tekarax", "vocab": 53, "width": 100, "norm": {"eps": 1e-5},
          "loop": {"start": 0, "stop": 2, "times": 2},
          "layers": [
              wkv(3, 10, 5, moe(4, 3, 20, shared=12)),
              latent(2, 12, 10, 20, 0.25, 1000, dense(36)),
              attention(5, 5, 12, 14, 0.3, rot(300.0, 4, (2.0, 1.0, 3.0, 16)), dense(28)),
          ]},
}


def _all_experts(case: dict) -> dict:
    case = copy.deepcopy(case)
    for entry in case["layers"]:
        if entry["mlp"] is not None and entry["mlp"]["kind"] == "moe":
            entry["mlp"]["router"]["top"] = entry["mlp"]["router"]["experts"]
    return case


# "Pa", "Qa", ...: the same models with EVERY expert chosen.  Random routers have close calls: where two experts' scores
# lie within bfloat16 rounding of one another the bfloat16 engine may choose the other one, and that position, and
# through states and keys all behind it, then differs by a whole expert's output.  So the bfloat16 engine is compared on
# these (same tensors, no discrete choice), the float32 engine on the true routing at every position, and the choice
# itself is tested on given inputs in test_tekarax_parts_gpu.py.
CASES.update({name + "a": _all_experts(case) for name, case in list(CASES.items())})


def variant(name: str, dtype: str) -> str:
    return name if dtype == "float32" else name + "a"


def config_for(name: str):
    from torchlet_b200.config import TekaraxConfig

    return TekaraxConfig.from_dict(CASES[name])


def config_json(name: str) -> dict:
    """The case as a checkpoint's config.json holds it: the decay ranks come from the tensors."""
    out = copy.deepcopy(CASES[name])
    for layer in out["layers"]:
        layer["mixer"].pop("decay_rank", None)
    return out


@functools.lru_cache(maxsize=None)
def weights_for(name: str, seed: int = 0):
    """bfloat16-rounded random weights as float32 tensors by name (so that both engines and the plain implementation
    hold the same numbers).  Routers are drawn wider, so that the experts' scores lie apart; mixes, bonuses, decays,
    sinks, biases and the rows of the passes are drawn so that each counts."""
    from torchlet_b200.weights import random_tensors

    tensors = random_tensors(config_for(name), seed=900 + seed, std=0.1, norm_std=0.1, dtype="bfloat16")
    g = torch.Generator().manual_seed(1300 + seed)
    out = {}
    for k, v in tensors.items():
        v = v.float()
        noise = torch.randn(v.shape, generator=g)
        if k.endswith(".router"):
            v = v * 4
        elif ".mix.mu." in k:
            v = 0.5 + 0.3 * noise
        elif k.endswith(".w0"):
            v = -1.5 + noise
        elif k.endswith(".mix.u"):
            v = 0.8 * noise
        elif k.endswith(".sink"):
            v = 0.5 + noise
        elif k == "loop.step":
            v = 0.5 * noise
        elif k.endswith(".b"):
            v = 0.4 * noise
        elif k == "embed":
            v = noise
        out[k] = v.to(torch.bfloat16).float()
    return out


def make_ids(name: str, length: int, seed: int):
    g = torch.Generator().manual_seed(7000 + seed)
    return torch.randint(0, CASES[name]["vocab"], (length,), generator=g).tolist()


@functools.lru_cache(maxsize=None)
def plain_logits(name: str, length: int, seed: int):
    ids = make_ids(name, length, seed)
    w = {k: v.double() for k, v in weights_for(name).items()}
    return ids, plain_tekarax.forward(CASES[name], w, ids).float()


def make_model(name: str, dtype: str):
    from torchlet_b200.engine.loading import build_model

    return build_model(config_for(name), {k: v.to(torch.bfloat16) for k, v in weights_for(name).items()}, dtype)


def make_runner(name: str, dtype: str, num_pages: int = 64, slots: int = 4, page_size: int = 16, budget: int = 512,
                max_seq_len: int = 512, cuda_graph: bool = False):
    from torchlet_b200.config import EngineConfig
    from torchlet_b200.engine import ModelRunner

    engine = EngineConfig(dtype=dtype, max_decode_slots=slots, kv_block_size=page_size, max_num_blocks=num_pages,
                          max_seq_len=max_seq_len, max_num_batched_tokens=budget, cuda_graph=cuda_graph)
    return ModelRunner(make_model(name, dtype), engine)


def write_checkpoint(folder, name: str) -> None:
    import json

    from safetensors.torch import save_file

    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(config_json(name)))
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in weights_for(name).items()}, str(folder / "model.safetensors"))


def replay(runner, rid, ids, cuts, finish=True):
    """Feed ``ids`` of one request in portions of the given sizes, asking for every position's logits; returns
    [len(ids), vocab] on the CPU."""
    from torchlet_b200.engine import StepEntry

    assert sum(cuts) == len(ids)
    runner.admit(rid)
    out, start = [], 0
    for size in cuts:
        logits = runner.step([StepEntry(rid, ids[start:start + size], list(range(size)))])
        out.append(logits.cpu().clone())
        start += size
    if finish:
        runner.finish(rid)
        runner.cache.check()
    return torch.cat(out)


def assert_close(got, want, dtype: str, what: str = ""):
    """Row by row: the largest difference of a position's logits against the largest |logit| of THAT position."""
    assert got.shape == want.shape, f"{what}: shapes {tuple(got.shape)} and {tuple(want.shape)}"
    assert torch.isfinite(got).all(), f"{what}: not finite"
    got, want = got.reshape(-1, got.shape[-1]).double(), want.reshape(-1, want.shape[-1]).double()
    ratio = (got - want).abs().amax(dim=1) / want.abs().amax(dim=1)
    worst = int(ratio.argmax())
    if dtype == "bfloat16":
        # Behind the norm of a sub-layer's result only its direction counts.  At the first positions a state has rank one
        # or two and a head's output is one value vector times the scalar k . r: where that scalar is within bfloat16
        # rounding of zero its sign is a coin's toss.  Random weights have such positions; the float32 engine is held to
        # its tolerance at EVERY position of the same tests, the bfloat16 engine at nine in ten, and nowhere may it be
        # off by more than half of the largest logit.
        over = int((ratio > TOLERANCE[dtype]).sum())
        assert over <= max(1, ratio.numel() // 10) and ratio[worst] <= 0.5, (
            f"{what}: {over} of {ratio.numel()} rows over {TOLERANCE[dtype]:.1e}; worst row {worst}: {ratio[worst]:.3e}")
        return
    assert ratio[worst] <= TOLERANCE[dtype], f"{what}: row {worst}: {ratio[worst]:.3e} > {TOLERANCE[dtype]:.1e}"
