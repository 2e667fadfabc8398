"""Prefill and decode throughput of the Tekarax design at layer sizes that resemble a real model's, beside the closest
existing design of equal size: Numuzen (a linear recurrence with a decay per key channel beside an attention with a sink
and a gate, a norm in front of and behind every sub-layer, experts whose weights multiply their inputs; same width,
layers, heads and vocabulary).

    python -m torchlet_b200.benchmarks.tekarax [--size 2b|1b] [--layers N] [--prefill 2048] [--batch 8]
                                               [--context 2048] [--steps 32] [--kernels]

Random bfloat16 weights made on the GPU.  Prefill: one request's whole prompt in one step (CUDA events around the
step, best of three).  Decode: ``batch`` requests with ``context`` cached tokens, replayed from the captured decode
step.  ``--kernels`` also times the step of either model with each of its kernel classes replaced by nothing: the
difference is that class's cost in place, and the two models' like classes stand side by side.
"""
from __future__ import annotations

import argparse
import json

import torch

from ..config import NumuzenConfig, TekaraxConfig
from .dodonex import build, time_decode, time_prefill
from .fusolix import in_place_costs
from .numuzen import KERNEL_CLASSES as NUMUZEN_CLASSES
from .numuzen import numuzen_config

SIZES = {
    # width, dense ff, vocabulary, (heads, KV heads, key size, value size) of the attention, (heads, size, value size,
    # rank) of the latent attention, (heads, size, decay rank) of the time mixing
    "2b": (2048, 8192, 32768, (16, 4, 128, 128), (16, 128, 128, 512), (32, 64, 64)),
    "1b": (1024, 4096, 32768, (16, 4, 64, 64), (8, 64, 64, 256), (16, 64, 32)),
}


def tekarax_config(size: str, layers: int, experts: int = 8, top: int = 2, window: int = 1024) -> dict:
    """Layers in the pattern time mixing, attention, time mixing, latent attention, ...; a feed-forward of ``experts``
    experts of which a token uses ``top``, each 1 / top as wide as the dense unit, with a shared expert a quarter as wide;
    every fourth layer has the dense unit."""
    width, ff, vocab, (H, G, d, dv), (LH, LD, LV, rank), (RH, RD, decay) = SIZES[size]
    attention = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": d ** -0.5,
                 "rot": {"base": 500000.0, "dims": d, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    latent = {"heads": LH, "dim": LD, "vdim": LV, "kv_rank": rank, "scale": LD ** -0.5, "mask": {"size": window}}
    mixing = {"heads": RH, "dim": RD, "decay_rank": decay}
    mixers = (("wkv", mixing), ("attention", attention), ("wkv", mixing), ("latent_attention", latent))
    routed = {"kind": "moe", "expert": {"ff": ff // top}, "router": {"experts": experts, "top": top}, "shared": {"ff": ff // 4}}
    out = [{"type": mixers[i % 4][0], "mixer": mixers[i % 4][1], "mlp": {"kind": "dense", "ff": ff} if i % 4 == 2 else routed}
           for i in range(layers)]
    return {"architecture": "Tekarax", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "layers": out}


KERNEL_CLASSES = {
    "time mixing (shift, decay, scan, norm and gate)": ("token_shift", "time_mixing_step", "gla_decay", "gla_scan", "gla_finish"),
    "attention (rotations, cache write, turning back and head gates)": ("normed_qk_store", "head_finish"),
    "attention (scores and values)": ("attention_tc", "attention_mma", "attention_generic"),
    "latent attention (prepare, absorb, scores and values, expand)":
        ("latent_prepare", "latent_absorb_q", "latent_attention_mma", "latent_attention", "latent_expand_o"),
    "routing (route, plan, scatter, combine)": ("moe_route", "moe_plan", "moe_scatter", "moe_combine"),
    "expert products": ("gemm_tc_grouped", "moe_gemm_simt"),
    "ends of sub-layers (zero, gate, norm behind, residual sum, next norm)": ("fill_zero", "residual_norm"),
}


def run(size: str = "2b", layers: int = 8, prefill: int = 2048, batch: int = 8, context: int = 2048, steps: int = 32,
        kernels: bool = False, experts: int = 8, top: int = 2, window: int = 1024) -> dict:
    record = {"workload": "tekarax", "size": size, "layers": layers, "prefill_tokens": prefill, "batch": batch,
              "context": context, "experts": experts, "top": top, "window": window}
    numuzen_classes = dict(NUMUZEN_CLASSES)
    numuzen_classes["attention (scores and values)"] = KERNEL_CLASSES["attention (scores and values)"]
    numuzen_classes["side stream (zero, norm behind the sub-layer)"] = ("fill_zero", "rms_scaled_add", "rms_scaled_add_partials")
    models = (("tekarax", TekaraxConfig.from_dict(tekarax_config(size, layers, experts, top, window)), KERNEL_CLASSES),
              ("numuzen_equal_size", NumuzenConfig.from_dict(numuzen_config(size, layers, experts, top, window)), numuzen_classes))
    for name, config, classes in models:
        model = build(config, seed=9)
        ms = time_prefill(model, prefill)
        us = time_decode(model, batch, context, steps)
        record[name] = {"prefill_ms": round(ms, 3), "prefill_tok_s": round(prefill / ms * 1e3, 1),
                        "decode_us": round(us, 1), "decode_tok_s": round(batch / us * 1e6, 1)}
        if kernels:
            record[name]["in_place_costs"] = in_place_costs(model, classes, ms, us, prefill, batch, context, steps)
        del model
        torch.cuda.empty_cache()
    record["value"] = record["tekarax"]["decode_tok_s"]
    record["unit"] = "tok/s"
    record["metric"] = f"decode tokens per second, batch {batch}, context {context}"
    return record


def main(argv=None) -> int:
    parser = argparse.ArgumentParser(description=__doc__.split("\n\n")[0])
    parser.add_argument("--size", choices=sorted(SIZES), default="2b")
    parser.add_argument("--layers", type=int, default=8)
    parser.add_argument("--prefill", type=int, default=2048)
    parser.add_argument("--batch", type=int, default=8)
    parser.add_argument("--context", type=int, default=2048)
    parser.add_argument("--steps", type=int, default=32)
    parser.add_argument("--experts", type=int, default=8)
    parser.add_argument("--top", type=int, default=2)
    parser.add_argument("--window", type=int, default=1024)
    parser.add_argument("--kernels", action="store_true")
    parser.add_argument("--only", choices=["prefill", "decode"], default=None,
                        help="one step of the Tekarax model alone, untimed (for a launch list)")
    args = parser.parse_args(argv)
    if args.only:
        model = build(TekaraxConfig.from_dict(tekarax_config(args.size, args.layers, args.experts, args.top, args.window)), seed=9)
        if args.only == "prefill":
            print(json.dumps({"prefill_ms": time_prefill(model, args.prefill, repeats=1)}))
        else:
            print(json.dumps({"decode_us": time_decode(model, args.batch, args.context, 2, warmup=1)}))
        return 0
    print(json.dumps(run(args.size, args.layers, args.prefill, args.batch, args.context, args.steps, args.kernels,
                         args.experts, args.top, args.window)))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
