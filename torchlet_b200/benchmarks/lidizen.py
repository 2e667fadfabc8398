"""Prefill and decode throughput of the Lidizen design at layer sizes that resemble a real model's, beside the closest
existing designs of equal size: Numuzen with attention layers only (a windowed softmax attention with q and k normed over the
whole projection, routed experts) and Fusolix (several residual streams read and written around every sub-layer, a windowed
attention, dense and routed feed-forwards in turn); same width, layers, heads, window and vocabulary.

    python -m torchlet_b200.benchmarks.lidizen [--size 2b|1b] [--layers N] [--prefill 2048] [--batch 8]
                                               [--context 2048] [--steps 32] [--kernels]

Random bfloat16 weights made on the GPU.  Prefill: one request's whole prompt in one step (CUDA events around the step, best
of three).  Decode: ``batch`` requests with ``context`` cached tokens, replayed from the captured decode step.  ``--kernels``
also times the step of every model with each of its kernel classes replaced by nothing: the difference is that class's cost
in place, and like classes stand side by side.
"""
from __future__ import annotations

import argparse
import json

import torch

from ..config import FusolixConfig, LidizenConfig, NumuzenConfig
from .dodonex import build, time_decode, time_prefill
from .fusolix import KERNEL_CLASSES as FUSOLIX_CLASSES
from .fusolix import fusolix_config, in_place_costs
from .numuzen import numuzen_config

SIZES = {
    # width, dense ff, vocabulary, heads, KV heads, key size, value size
    "2b": (2048, 8192, 32768, 16, 4, 128, 128),
    "1b": (1024, 4096, 32768, 16, 4, 64, 64),
}


def lidizen_config(size: str, layers: int, experts: int = 8, top: int = 2, window: int = 1024, keep: int = 64,
                   streams: int = 4, kv_heads: int | None = None) -> dict:
    """The feed-forward alternates between the dense unit and ``experts`` experts of which a token uses ``top``, each 1 / top
    as wide; every layer's values are mixed with the first one's."""
    width, ff, vocab, H, G, d, dv = SIZES[size]
    mixer = {"heads": H, "kv_heads": kv_heads or G, "dim": d, "vdim": dv, "scale": d ** -0.5, "v_mix": True,
             "mask": {"size": window, "keep_first": keep}, "rot": {"base": 1000000.0, "dims": d // 2}}
    routed = {"kind": "moe", "expert": {"ff": ff // top}, "router": {"experts": experts, "top": top}}
    out = [{"type": "attention", "mixer": mixer, "mlp": routed if i % 2 else {"kind": "dense", "ff": ff}} for i in range(layers)]
    return {"architecture": "Lidizen", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": 1e-6},
            "embedding": {"bigram": {"buckets": 65521, "mul_prev": 8191, "mul_cur": 127}}, "layers": out}


def numuzen_attention_config(size: str, layers: int, experts: int = 8, top: int = 2, window: int = 1024,
                             kv_heads: int | None = None) -> dict:
    raw = numuzen_config(size, 2 * layers, experts, top, window)
    raw["layers"] = [layer for layer in raw["layers"] if layer["type"] == "attention"]
    for layer in raw["layers"]:
        layer["mixer"]["kv_heads"] = kv_heads or layer["mixer"]["kv_heads"]
    return raw


KERNEL_CLASSES = {
    "token, pair row, norm, streams": ("token_embed",),
    "attention (norm, rotation, score and value mixing, cache write)": ("qkv_prepare",),
    "attention (scores and values)": ("attention_spread", "attention_mixed_decode", "attention_generic"),
    "streams (read and norm, write)": ("hyper_read_norm", "hyper_write", "hyper_collapse"),
    "routing (route, plan, scatter, combine)": ("moe_route", "moe_plan", "moe_scatter", "moe_combine"),
    "expert products": ("gemm_tc_grouped", "moe_gemm_simt"),
    "gated product of the dense unit": ("gemm_tc_gated",),
}

NUMUZEN_CLASSES = {
    "attention (norm, rotation, cache write)": ("normed_qk_store",),
    "attention (scores and values)": ("attention_tc", "attention_mma", "attention_generic"),
    "side stream (zero, norm behind the sub-layer)": ("fill_zero", "rms_scaled_add", "rms_scaled_add_partials", "residual_norm"),
    "routing (route, plan, scatter, combine)": ("moe_route", "moe_plan", "moe_scatter", "moe_combine"),
    "expert products": ("gemm_tc_grouped", "moe_gemm_simt"),
}


def run(size: str = "2b", layers: int = 8, prefill: int = 2048, batch: int = 8, context: int = 2048, steps: int = 32,
        kernels: bool = False, experts: int = 8, top: int = 2, window: int = 1024, keep: int = 64, streams: int = 4) -> dict:
    record = {"workload": "lidizen", "size": size, "layers": layers, "prefill_tokens": prefill, "batch": batch,
              "context": context, "experts": experts, "top": top, "window": window, "keep_first": keep, "streams": streams}
    models = (
        ("lidizen", LidizenConfig.from_dict(lidizen_config(size, layers, experts, top, window, keep, streams)), KERNEL_CLASSES),
        ("numuzen_attention_equal_size", NumuzenConfig.from_dict(numuzen_attention_config(size, layers, experts, top, window)),
         NUMUZEN_CLASSES),
        ("fusolix_equal_size", FusolixConfig.from_dict(fusolix_config(size, layers, experts, top, window, streams=streams)),
         FUSOLIX_CLASSES))
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
    record["value"] = record["lidizen"]["decode_tok_s"]
    record["unit"] = "tok/s"
    record["metric"] = f"decode tokens per second, batch {batch}, context {context}"
    return record


def main(argv=None) -> int:
    parser = argparse.ArgumentParser(description=__doc__.split("\n\n")[0])
    parser.add_argument("--size", choices=sorted(SIZES), default="2b")
    for name, value in (("layers", 8), ("prefill", 2048), ("batch", 8), ("context", 2048), ("steps", 32), ("experts", 8),
                        ("top", 2), ("window", 1024), ("keep", 64), ("streams", 4)):
        parser.add_argument(f"--{name}", type=int, default=value)
    parser.add_argument("--kv-heads", type=int, default=None, help="with --only: another number of KV heads")
    parser.add_argument("--kernels", action="store_true")
    parser.add_argument("--only", choices=["prefill", "decode"], default=None,
                        help="one step of one model alone, untimed (for a launch list)")
    parser.add_argument("--model", choices=["lidizen", "numuzen"], default="lidizen", help="which one with --only")
    args = parser.parse_args(argv)
    if args.only:
        common = (args.size, args.layers, args.experts, args.top, args.window)
        if args.model == "lidizen":
            config = LidizenConfig.from_dict(lidizen_config(*common, args.keep, args.streams, args.kv_heads))
        else:
            config = NumuzenConfig.from_dict(numuzen_attention_config(*common, args.kv_heads))
        model = build(config, seed=9)
        if args.only == "prefill":
            print(json.dumps({"prefill_ms": time_prefill(model, args.prefill, repeats=1)}))
        else:
            print(json.dumps({"decode_us": time_decode(model, args.batch, args.context, 2, warmup=1)}))
        return 0
    print(json.dumps(run(args.size, args.layers, args.prefill, args.batch, args.context, args.steps, args.kernels,
                         args.experts, args.top, args.window, args.keep, args.streams)))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
