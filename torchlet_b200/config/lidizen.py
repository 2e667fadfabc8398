"""Typed configuration of the Lidizen design: a decoder-only model whose layers are listed one by one in
``config.json``.

    {"architecture": "Lidizen", "vocab": V, "width": W, "streams": n, "norm": {"eps": e},
     "embedding": {"bigram": {"buckets", "mul_prev", "mul_cur"}},
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "v_mix", "mask": {"size", "keep_first"},
                           "rot": {"base", "dims"}},
                 "mlp": {"kind": "dense", "ff"}
                      | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}} | null}, ...]}

The token's embedding row and a row of the table ``bigram``, chosen by the token and the one before it, are summed and
pass a layer norm (``embed.norm``); ``streams`` copies of the result are the residual streams (hyper-connections:
``l<i>.hc1.*`` for the mixer, ``l<i>.hc2.*`` for the feed-forward).  Norms are layer norms with a weight and no bias
(``l<i>.norm1``, ``l<i>.norm2``).  The mixer ``l<i>.mix.*``: an attention with biases, q and k normed over the whole
projection, an interleaved partial rotation, scores mixed across the heads, a sliding window beside which the first
``keep_first`` tokens stay visible, and values that are mixed with those of the first layer that has ``v_mix``.  The
feed-forward ``l<i>.mlp.*``: a silu-gated unit with biases, or a mixture of ungated experts with the square of relu
whose router has a bias and weighs the chosen experts by the softmax over their logits alone.  Output: the embedding
table behind the layer norm ``final.norm``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Optional

from .registry import register_architecture
from .spec import LayerSpec, ModelSpec, NormSlot, PartSpec, ScheduleEntry, TokenPairs

DEFAULT_MAX_POSITIONS = 1 << 17  # the design has no position limit of its own; the engine wants a bound


def _positive_int(value, what: str) -> int:
    if not isinstance(value, int) or isinstance(value, bool) or value <= 0:
        raise ValueError(f"{what} must be a positive integer, got {value!r}")
    return value


def _need(mapping, keys, what: str) -> None:
    if not isinstance(mapping, dict):
        raise ValueError(f"{what} must be an object")
    missing = [key for key in keys if key not in mapping]
    if missing:
        raise ValueError(f"{what} lacks {', '.join(missing)}")


def _check_attention(mixer, what: str) -> None:
    _need(mixer, ("heads", "kv_heads", "dim", "vdim", "scale"), what)
    for key in ("heads", "kv_heads", "dim", "vdim"):
        _positive_int(mixer[key], f"{what}.{key}")
    if mixer["heads"] % mixer["kv_heads"]:
        raise ValueError(f"{what}: heads {mixer['heads']} is no multiple of kv_heads {mixer['kv_heads']}")
    rot = mixer.get("rot")
    if rot is not None:
        _need(rot, ("base", "dims"), f"{what}.rot")
        if not isinstance(rot["dims"], int) or rot["dims"] % 2 or not 0 < rot["dims"] <= mixer["dim"]:
            raise ValueError(f"{what}.rot.dims {rot['dims']!r} must be even and at most dim {mixer['dim']}")
    mask = mixer.get("mask")
    if mask is not None:
        _need(mask, ("size",), f"{what}.mask")
        _positive_int(mask["size"], f"{what}.mask.size")
        if int(mask.get("keep_first", 0)) < 0:
            raise ValueError(f"{what}.mask.keep_first must not be negative")


def _check_mlp(mlp, what: str) -> None:
    kind = mlp.get("kind") if isinstance(mlp, dict) else None
    if kind == "dense":
        _need(mlp, ("ff",), what)
        _positive_int(mlp["ff"], f"{what}.ff")
    elif kind == "moe":
        _need(mlp, ("expert", "router"), what)
        _need(mlp["expert"], ("ff",), f"{what}.expert")
        _need(mlp["router"], ("experts", "top"), f"{what}.router")
        _positive_int(mlp["expert"]["ff"], f"{what}.expert.ff")
        experts = _positive_int(mlp["router"]["experts"], f"{what}.router.experts")
        if _positive_int(mlp["router"]["top"], f"{what}.router.top") > experts:
            raise ValueError(f"{what}: router.top {mlp['router']['top']} exceeds router.experts {experts}")
    else:
        raise ValueError(f"{what}: unknown kind {kind!r} (known: dense, moe)")


@register_architecture("Lidizen")
@dataclass(frozen=True)
class LidizenConfig:
    vocab: int
    width: int
    layers: tuple  # of dicts as in config.json: type, mixer, mlp
    streams: int = 1
    norm_eps: float = 1e-6
    bigram: Optional[tuple] = None  # (buckets, mul_prev, mul_cur); None: no table of token pairs
    max_position_embeddings: int = DEFAULT_MAX_POSITIONS
    eos_token_id: Optional[int] = None

    architecture = "Lidizen"

    def __post_init__(self) -> None:
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        _positive_int(self.streams, "streams")
        if not self.norm_eps > 0:
            raise ValueError("norm.eps must be positive")
        if self.bigram is not None:
            _positive_int(self.bigram[0], "embedding.bigram.buckets")
        if not self.layers:
            raise ValueError("'layers' is empty")
        shared = None  # (kv_heads, vdim) of the layers whose values are mixed
        for i, layer in enumerate(self.layers):
            if layer.get("type") != "attention":
                raise ValueError(f"layer {i}: unknown type {layer.get('type')!r} (known: attention)")
            mixer = layer.get("mixer")
            _check_attention(mixer, f"layer {i}: mixer")
            if mixer.get("v_mix"):
                mine = (mixer["kv_heads"], mixer["vdim"])
                if shared is not None and shared != mine:
                    raise ValueError(f"layer {i}: values of {mine[0]} x {mine[1]} cannot be mixed with the first such "
                                     f"layer's, which are {shared[0]} x {shared[1]}")
                shared = mine
            if layer.get("mlp") is not None:
                _check_mlp(layer["mlp"], f"layer {i}: mlp")

    # ------------------------------------------------------------------ io
    @classmethod
    def from_dict(cls, raw: dict) -> "LidizenConfig":
        missing = [key for key in ("vocab", "width", "layers") if key not in raw]
        if missing:
            raise ValueError(f"config.json lacks required keys: {', '.join(missing)}")
        bigram = (raw.get("embedding") or {}).get("bigram")
        if bigram is not None:
            _need(bigram, ("buckets", "mul_prev", "mul_cur"), "embedding.bigram")
            bigram = (int(bigram["buckets"]), int(bigram["mul_prev"]), int(bigram["mul_cur"]))
        values = dict(vocab=raw["vocab"], width=raw["width"], layers=tuple(copy.deepcopy(list(raw["layers"]))),
                      streams=int(raw.get("streams", 1)), norm_eps=float((raw.get("norm") or {}).get("eps", 1e-6)),
                      bigram=bigram, eos_token_id=raw.get("eos_token_id"))
        if raw.get("max_position_embeddings") is not None:
            values["max_position_embeddings"] = int(raw["max_position_embeddings"])
        return cls(**values)

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
               "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(list(self.layers))}
        if self.bigram is not None:
            out["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), self.bigram))}
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            out["max_position_embeddings"] = self.max_position_embeddings
        if self.eos_token_id is not None:
            out["eos_token_id"] = self.eos_token_id
        return out

    # ------------------------------------------------------------ structure
    def _mixer(self, m: dict, value_mix: Optional[str]) -> PartSpec:
        rot, mask = m.get("rot"), m.get("mask") or {}
        positions = None
        if rot is not None:
            positions = PartSpec("rotary_partial", {"head_dim": int(m["dim"]), "dims": int(rot["dims"]),
                                                    "base": float(rot["base"]), "scaling": None, "pairing": "interleaved"})
        return PartSpec("gated_attention", {
            "hidden_size": self.width, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]),
            "head_dim": int(m["dim"]), "v_dim": int(m["vdim"]), "scale": float(m["scale"]), "bias": True,
            "qk_norm": "whole", "eps": self.norm_eps, "positions": positions, "score_mix": True, "value_mix": value_mix,
            "window": int(mask["size"]) if mask.get("size") else None, "keep_first": int(mask.get("keep_first", 0) or 0)})

    def _feed_forward(self, mlp: Optional[dict]) -> Optional[PartSpec]:
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return PartSpec("gated_mlp", {"hidden_size": self.width, "intermediate_size": int(mlp["ff"]),
                                          "activation": "silu", "bias": True})
        return PartSpec("routed_clamped_glu", {
            "hidden_size": self.width, "intermediate_size": int(mlp["expert"]["ff"]), "unit": "relu_squared",
            "num_experts": int(mlp["router"]["experts"]), "top_k": int(mlp["router"]["top"]), "score": "chosen_softmax",
            "router_bias": True, "weight_on": "output"})

    def model_spec(self) -> ModelSpec:
        W = self.width
        norm = PartSpec("layer_norm", {"size": W, "eps": self.norm_eps, "weight_name": "", "bias_name": None})
        layers, schedule, mixed_before = [], [], False
        for i, layer in enumerate(self.layers):
            value_mix = None
            if layer["mixer"].get("v_mix"):
                value_mix = "later" if mixed_before else "first"
                mixed_before = True
            feed_forward = self._feed_forward(layer.get("mlp"))
            norms, unused = [NormSlot("mixer_norm", norm, "norm1")], ()
            if feed_forward is not None:
                norms.append(NormSlot("feed_forward_norm", norm, "norm2"))
            else:  # a checkpoint may carry the second sub-layer's norm and connections all the same
                n = self.streams
                unused = (("norm2", (W,)), ("hc2.in", (n,)), ("hc2.out", (n,)), ("hc2.mix", (n, n)))
            layers.append(LayerSpec(
                prefix=f"l{i}.", block="hyper_connected", mixer=self._mixer(layer["mixer"], value_mix),
                feed_forward=feed_forward, norms=tuple(norms), mixer_prefix="mix.", feed_forward_prefix="mlp.",
                block_params={"streams": self.streams, "taps": None, "connections": ("hc1.", "hc2."), "unused": unused}))
            schedule.append(ScheduleEntry(layer=i))
        pairs = TokenPairs("bigram", *self.bigram) if self.bigram is not None else None
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=W,
            max_position_embeddings=self.max_position_embeddings, embedding_name="embed",
            layers=tuple(layers), schedule=tuple(schedule), final_norm=norm, final_norm_prefix="final.norm",
            lm_head_name="lm_head", tie_word_embeddings=True, streams=self.streams, embedding_norm=norm,
            embedding_norm_prefix="embed.norm", token_pairs=pairs)
        spec.validate()
        return spec
