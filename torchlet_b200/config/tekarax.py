"""Typed configuration of the Tekarax design: a decoder-only model whose layers are listed one by one in
``config.json``, a stretch of which may run several times.

    {"architecture": "Tekarax", "vocab": V, "width": W, "norm": {"eps": e},
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale",
                           "rot": {"base", "dims", "scaling": {"factor", "low", "high", "original"}}}, "mlp": ...},
                {"type": "latent_attention",
                 "mixer": {"heads", "dim", "vdim", "kv_rank", "scale", "mask": {"size"}}, "mlp": ...},
                {"type": "wkv", "mixer": {"heads", "dim"}, "mlp": ...}]}
    mlp: {"kind": "dense", "ff"} | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"},
          "shared": {"ff"} or absent} | null

Every layer is a sandwich of layer norms (a weight, no bias) around its two sub-layers, each of whose results is
multiplied by a sigmoid gate of its own input before the norm behind it: x += norm1b(mixer(h) * sigmoid(rg1 h + rg1.b)),
h = norm1(x), and the same with norm2, norm2b, rg2 and the feed-forward.  Layers ``loop.start .. loop.stop - 1`` run
``loop.times`` times in a row with the same weights and a cache or state of their own each time; before pass t, the first
included, row t of ``loop.step`` is added to the stream.  The mixers: an attention with rotated values, a learned sink
and one sigmoid gate a head; a latent attention without positions over a sliding window; and a time-mixing recurrence
with token shift, a data-dependent decay and a bonus for the current token.  The feed-forward is an ungated unit with the
square of relu and biases, or a mixture of silu-gated experts: sigmoid scores, not renormalized, which multiply the
chosen experts' inputs, and an always-on shared expert.  Output: ``head`` behind the layer norm ``final.norm``.
One size stands in no key: the decay rank of a "wkv" layer is the number of rows of its ``l<i>.mix.w1``
(``with_tensor_shapes``), or the mixer's ``decay_rank``.
"""
from __future__ import annotations

import copy
import dataclasses
from dataclasses import dataclass
from typing import Optional

from .registry import register_architecture
from .spec import LayerSpec, ModelSpec, NormSlot, PartSpec, ScheduleEntry

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


MIXER_SIZES = {
    "attention": ("heads", "kv_heads", "dim", "vdim"),
    "latent_attention": ("heads", "dim", "vdim", "kv_rank"),
    "wkv": ("heads", "dim"),
}
MIXER_OTHERS = {"attention": ("scale", "rot"), "latent_attention": ("scale", "mask"), "wkv": ()}


def _check_mixer(kind: str, m: dict, what: str) -> None:
    _need(m, MIXER_SIZES[kind] + MIXER_OTHERS[kind], what)
    for key in MIXER_SIZES[kind]:
        _positive_int(m[key], f"{what}.{key}")
    if kind == "latent_attention":
        _need(m["mask"], ("size",), f"{what}.mask")
        _positive_int(m["mask"]["size"], f"{what}.mask.size")
    elif kind == "attention":
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"{what}: heads {m['heads']} is no multiple of kv_heads {m['kv_heads']}")
        if m["vdim"] % 2:
            raise ValueError(f"{what}: values of {m['vdim']} entries cannot turn in pairs")
        rot = m["rot"]
        _need(rot, ("base", "dims"), f"{what}.rot")
        if not isinstance(rot["dims"], int) or rot["dims"] % 2 or not 0 < rot["dims"] <= m["dim"]:
            raise ValueError(f"{what}.rot.dims {rot['dims']!r} must be even and at most {m['dim']}")
        if rot.get("scaling") is not None:
            _need(rot["scaling"], ("factor", "low", "high", "original"), f"{what}.rot.scaling")


def _check_mlp(mlp: dict, what: str) -> None:
    if mlp.get("kind") == "dense":
        _positive_int(mlp.get("ff"), f"{what}.ff")
    elif mlp.get("kind") == "moe":
        _need(mlp, ("expert", "router"), what)
        _need(mlp["expert"], ("ff",), f"{what}.expert")
        _need(mlp["router"], ("experts", "top"), f"{what}.router")
        _positive_int(mlp["expert"]["ff"], f"{what}.expert.ff")
        experts = _positive_int(mlp["router"]["experts"], f"{what}.router.experts")
        if _positive_int(mlp["router"]["top"], f"{what}.router.top") > experts:
            raise ValueError(f"{what}: router.top {mlp['router']['top']} does not fit {experts} experts")
        if mlp.get("shared") is not None:
            _positive_int(mlp["shared"].get("ff"), f"{what}.shared.ff")
    else:
        raise ValueError(f"{what}: unknown kind {mlp.get('kind')!r} (known: dense, moe)")


@register_architecture("Tekarax")
@dataclass(frozen=True)
class TekaraxConfig:
    vocab: int
    width: int
    layers: tuple  # of dicts as in config.json: type, mixer, mlp
    norm_eps: float = 1e-6
    loop: Optional[tuple] = None  # (start, stop, times)
    max_position_embeddings: int = DEFAULT_MAX_POSITIONS
    eos_token_id: Optional[int] = None

    architecture = "Tekarax"

    def __post_init__(self) -> None:
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        if not self.norm_eps > 0:
            raise ValueError("norm.eps must be positive")
        if not self.layers:
            raise ValueError("'layers' is empty")
        if self.loop is not None:
            start, stop, times = self.loop
            if not (isinstance(start, int) and isinstance(stop, int) and 0 <= start < stop <= len(self.layers)):
                raise ValueError(f"loop: layers {start} .. {stop} - 1 do not lie within the {len(self.layers)} layers")
            _positive_int(times, "loop.times")
        for i, layer in enumerate(self.layers):
            kind = layer.get("type")
            if kind not in MIXER_SIZES:
                raise ValueError(f"layer {i}: unknown type {kind!r} (known: {', '.join(sorted(MIXER_SIZES))})")
            _check_mixer(kind, layer.get("mixer"), f"layer {i}: mixer")
            if layer.get("mlp") is not None:
                _check_mlp(layer["mlp"], f"layer {i}: mlp")

    # ------------------------------------------------------------------ io
    @classmethod
    def from_dict(cls, raw: dict) -> "TekaraxConfig":
        missing = [key for key in ("vocab", "width", "layers") if key not in raw]
        if missing:
            raise ValueError(f"config.json lacks required keys: {', '.join(missing)}")
        loop = raw.get("loop")
        if loop is not None:
            _need(loop, ("start", "stop"), "loop")
            loop = (loop["start"], loop["stop"], loop.get("times", 1))
        values = dict(vocab=raw["vocab"], width=raw["width"], layers=tuple(copy.deepcopy(list(raw["layers"]))),
                      norm_eps=float((raw.get("norm") or {}).get("eps", 1e-6)), loop=loop,
                      eos_token_id=raw.get("eos_token_id"))
        if raw.get("max_position_embeddings") is not None:
            values["max_position_embeddings"] = int(raw["max_position_embeddings"])
        return cls(**values)

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(list(self.layers))}
        if self.loop is not None:
            out["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            out["max_position_embeddings"] = self.max_position_embeddings
        if self.eos_token_id is not None:
            out["eos_token_id"] = self.eos_token_id
        return out

    def with_tensor_shapes(self, shapes: dict) -> "TekaraxConfig":
        """The sizes that only the checkpoint gives: a wkv layer's decay rank is the number of rows of its ``w1``.
        ``shapes``: tensor name -> shape."""
        layers = copy.deepcopy(list(self.layers))
        for i, layer in enumerate(layers):
            name = f"l{i}.mix.w1"
            if layer["type"] == "wkv" and name in shapes and len(shapes[name]) == 2:
                layer["mixer"]["decay_rank"] = int(shapes[name][0])
        return dataclasses.replace(self, layers=tuple(layers))

    # ------------------------------------------------------------ structure
    def layer_runs(self) -> list:
        """The layers in the order they run: (layer, number of the pass that begins with it, or None)."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        start, stop, times = self.loop
        runs = [(i, None) for i in range(start)]
        for t in range(times):
            runs += [(i, t if i == start else None) for i in range(start, stop)]
        return runs + [(i, None) for i in range(stop, n)]

    def _mixer(self, i: int, kind: str, m: dict) -> PartSpec:
        W, eps = self.width, self.norm_eps
        if kind == "wkv":
            if not m.get("decay_rank"):
                raise ValueError(f"layer {i}: the decay rank is not known: it comes from the shape of l{i}.mix.w1 "
                                 "(with_tensor_shapes) or the mixer's 'decay_rank'")
            return PartSpec("time_mixing", {"hidden_size": W, "num_heads": int(m["heads"]), "head_dim": int(m["dim"]),
                                            "decay_rank": int(m["decay_rank"]), "eps": eps})
        if kind == "latent_attention":
            return PartSpec("latent_attention", {
                "hidden_size": W, "num_heads": int(m["heads"]), "head_dim": int(m["dim"]), "rot_dim": 0,
                "v_dim": int(m["vdim"]), "q_rank": None, "kv_rank": int(m["kv_rank"]), "scale": float(m["scale"]),
                "eps": eps, "window": int(m["mask"]["size"])})
        rot = m["rot"]
        base = float(rot["base"])
        scaling = dict(rot["scaling"]) if rot.get("scaling") else None
        keys = PartSpec("rotary_partial", {"head_dim": int(m["dim"]), "dims": int(rot["dims"]), "base": base, "scaling": scaling})
        values = PartSpec("rotary_partial", {"head_dim": int(m["vdim"]), "dims": int(m["vdim"]), "base": base})
        return PartSpec("gated_attention", {
            "hidden_size": W, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]), "head_dim": int(m["dim"]),
            "v_dim": int(m["vdim"]), "scale": float(m["scale"]), "positions": keys, "value_rotation": values,
            "sink": "learned", "gate": "head_sigmoid", "eps": eps})

    def _feed_forward(self, mlp: Optional[dict]) -> Optional[PartSpec]:
        W = self.width
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return PartSpec("mlp", {"hidden_size": W, "intermediate_size": int(mlp["ff"]), "activation": "relu_squared",
                                    "bias": True})
        shared = None
        if mlp.get("shared") is not None:
            shared = PartSpec("gated_mlp", {"hidden_size": W, "intermediate_size": int(mlp["shared"]["ff"]),
                                            "activation": "silu", "bias": False})
        return PartSpec("routed_clamped_glu", {
            "hidden_size": W, "intermediate_size": int(mlp["expert"]["ff"]), "limit": None,
            "num_experts": int(mlp["router"]["experts"]), "top_k": int(mlp["router"]["top"]), "score": "sigmoid",
            "renormalize": False, "weight_on": "input", "shared": shared, "shared_prefix": "shared."})

    def model_spec(self) -> ModelSpec:
        W = self.width
        norm = PartSpec("layer_norm", {"size": W, "eps": self.norm_eps, "weight_name": "", "bias_name": None})
        layers = []
        for i, layer in enumerate(self.layers):
            feed_forward = self._feed_forward(layer.get("mlp"))
            norms = [NormSlot("mixer_norm", norm, "norm1"), NormSlot("mixer_post_norm", norm, "norm1b")]
            if feed_forward is not None:
                norms += [NormSlot("feed_forward_norm", norm, "norm2"), NormSlot("feed_forward_post_norm", norm, "norm2b")]
            layers.append(LayerSpec(
                prefix=f"l{i}.", block="sandwich", mixer=self._mixer(i, layer["type"], layer["mixer"]),
                feed_forward=feed_forward, norms=tuple(norms), mixer_prefix="mix.", feed_forward_prefix="mlp.",
                block_params={"gates": ("rg1", "rg2")}))
        schedule = tuple(ScheduleEntry(layer=i, add_row=began) for i, began in self.layer_runs())
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=W,
            max_position_embeddings=self.max_position_embeddings, embedding_name="embed", layers=tuple(layers),
            schedule=schedule, final_norm=norm, final_norm_prefix="final.norm", lm_head_name="head",
            tie_word_embeddings=False, stream_rows_name="loop.step" if self.loop is not None else None,
            stream_rows=self.loop[2] if self.loop is not None else 0)
        spec.validate()
        return spec
