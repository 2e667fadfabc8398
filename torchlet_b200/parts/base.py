"""Interfaces of the parts a layer is put together from, and their registries.

A part knows its own sizes and constants (from its ``PartSpec``) and the names of
its own tensors below a prefix.  It does not know which model it is in, which layer
it is, or what stands before or after it.  The reference has the same parts as
``nn.Module`` classes with constructor arguments
(v10_triton_paged_gqa/layer/{gqa,ffn_swiglu,rms_norm,rope,transformer_block}.py);
here each kind is looked up by name so that a layer may choose any of them.

Data contract of a step (``StepContext`` in ``torchlet_b200.engine.batch``):

* ``x``   : the normed input of a sub-layer, ``[T, hidden]`` in the compute dtype;
* ``acc`` : the residual stream, ``[T, hidden]`` in float32.  A mixer or a
  feed-forward ADDS its output into ``acc``; the residual sum is therefore always
  taken in 32-bit.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Optional

from ..config.spec import PartSpec


@dataclass(frozen=True)
class TensorSpec:
    """A tensor a part expects in the checkpoint."""

    name: str
    shape: tuple
    # "normal": N(0, std); "ones": 1 + N(0, norm_std); "zeros": N(0, norm_std); "eye": identity + N(0, norm_std)
    init: str = "normal"
    optional: bool = False


@dataclass(frozen=True)
class KVSpec:
    """Per-token history a mixer keeps in pages: keys and values of every token,
    or of the last ``window`` tokens only.  ``planes`` is how many rows of ``head_dim`` a token
    keeps per KV head: 2 (a key and a value), or 1 for a mixer whose keys and values are
    expanded from one cached row (a latent).  ``keep_first``: beside the window, the first that many
    tokens of a sequence stay (their pages are never given back while the request lives)."""

    num_kv_heads: int
    head_dim: int
    window: Optional[int] = None
    planes: int = 2
    keep_first: int = 0

    def group_key(self) -> tuple:
        key = (self.num_kv_heads, self.head_dim, self.window, self.planes)
        return key + (self.keep_first,) if self.keep_first and self.window is not None else key


@dataclass(frozen=True)
class StateSpec:
    """Fixed-size state a part keeps per live request (one row per slot), zeroed when a request is
    admitted.  ``per_tokens`` = P: the state is one ``shape`` entry for every P tokens of the longest
    sequence the engine admits, ``[ceil(max_seq_len / P), *shape]`` a slot (a summary row per block of
    tokens, for instance)."""

    shape: tuple
    dtype: str = "float32"
    per_tokens: Optional[int] = None

    def slot_shape(self, max_seq_len: int) -> tuple:
        if self.per_tokens is None:
            return tuple(self.shape)
        return (-(-max_seq_len // self.per_tokens), *self.shape)


class Part:
    """Base of all parts.  Sub-classes set ``kind`` and implement what applies."""

    kind: str = ""

    def __init__(self, spec: PartSpec):
        self.spec = spec

    @classmethod
    def expected_tensors(cls, spec: PartSpec, prefix: str) -> list[TensorSpec]:
        return []

    def load(self, tensors: dict, prefix: str, device, dtype) -> None:
        """Take this part's tensors (by full name) and lay them out for its kernels."""


class Norm(Part):
    """A norm reads rows of the float32 stream ``acc`` and returns them normed in the compute
    dtype.  A sub-class implements ``forward``; blocks and the model call ``apply``, which first
    completes any sum into ``acc`` that a product left unfinished, so that ``forward`` can read
    ``acc`` as it stands.  A norm that can take over such a sum and finish it inside its own
    kernel sets ``fuses_pending`` and asks ``ctx.take_pending(acc)`` itself."""

    fuses_pending = False

    def apply(self, ctx, acc, out=None, rows=None, name="normed"):
        if rows is None and self.residual_terms() is not None:
            residual = ctx.take_residual(acc)
            if residual is not None:  # the end of the sub-layer before and this norm as one kernel
                if out is None:
                    out = ctx.buffer(name, tuple(acc.shape), ctx.dtype)
                residual.finish(self.residual_terms() + (out,))
                return out
        if not self.fuses_pending:
            ctx.flush_pending()
        return self.forward(ctx, acc, out=out, rows=rows, name=name)

    def residual_terms(self):
        """(weight, bias or None, eps, centre) of a norm over whole rows that may join the end of the sub-layer before it
        in one kernel (``ops.residual_norm``); None: not such a norm."""
        return None

    def forward(self, ctx, acc, out=None, rows=None, name="normed"):
        """Return the normed ``acc`` rows (all, or those ``rows`` names, int32) in the compute
        dtype; ``out`` or a buffer called ``name`` receives them."""
        raise NotImplementedError

    def add_normed(self, ctx, y, acc, m: float = 1.0, clear: bool = False, gate=None) -> None:
        """acc += m * norm(y) in float32, for a norm that stands BEHIND a sub-layer (``y`` is the
        float32 side stream the sub-layer added its output into; ``clear``: and leave y zeroed).
        ``gate`` = (float32 rows or split sums of them, splits or 0, bias or None): y is multiplied by
        sigmoid(gate) first.  The sum may be left to the next norm of ``acc`` (``ctx.leave_residual``)."""
        terms = self.residual_terms()
        if terms is None:
            raise NotImplementedError(f"the norm {self.kind!r} cannot stand behind a sub-layer")
        pending = ctx.take_pending(y)
        if pending is None:
            ctx.flush_pending()
        ctx.leave_residual(acc, y, terms, m, clear, pending, gate)


class Positions(Part):
    """A position encoding applied inside a mixer: ``encode(ctx, qkv, num_heads, num_kv_heads)``
    changes the q and k heads of the fused ``qkv`` rows in place; the mixer then stores k and v
    itself.  An encoding that can write k and v to the cache pages in the same pass sets
    ``stores_kv`` and implements ``encode_and_store(ctx, qkv, num_heads, num_kv_heads, cache)``
    instead.  ``graph_safe`` False keeps a model that uses it out of the captured decode graph
    (it plans on the host)."""

    graph_safe = True
    stores_kv = False

    def encode(self, ctx, qkv, num_heads, num_kv_heads) -> None:
        raise NotImplementedError


class Mixer(Part):
    def kv_spec(self) -> Optional[KVSpec]:
        return None

    def state_spec(self):
        """None, one ``StateSpec``, or a dict name -> ``StateSpec`` for a mixer that keeps several
        states (``cache.state`` is then a dict of tensors under the same names)."""
        return None

    def forward(self, ctx, x, acc, cache) -> None:
        """Mix ``x`` over each request's history and add the result into ``acc``.

        ``cache`` is the ``LayerCache`` of this execution: pages and block table if
        ``kv_spec`` is set, the state rows if ``state_spec`` is set, and
        ``cache.writable`` False when the execution reads another's cache.
        """
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, ctx, x, acc) -> None:
        """Add the feed-forward of ``x`` into ``acc``."""
        raise NotImplementedError


class TokenInput(Part):
    """Something added to the stream after a layer's sub-layers that is computed from the
    step's token ids themselves (``ctx.tokens``) and the stream."""

    def forward(self, ctx, acc, m: float = 1.0) -> None:
        """acc += m * f(acc, tokens)."""
        raise NotImplementedError


class Block:
    """An arrangement of a layer's parts around the residual stream.  ``norm_roles`` names the
    norms the arrangement needs; the layer's description must hold one for each role, and
    ``norms`` maps the roles to the built parts.  ``feed_forward`` and ``token_input`` may be
    None; ``params`` are the arrangement's own constants from the layer's description."""

    kind: str = ""
    norm_roles: tuple = ()

    def __init__(self, mixer: Mixer, feed_forward: Optional[FeedForward], norms: dict, params: Optional[dict] = None,
                 token_input: Optional[TokenInput] = None):
        missing = [role for role in self.norm_roles if role not in norms]
        if missing:
            raise ValueError(f"block arrangement {self.kind!r} needs norms for the roles {missing}")
        self.mixer = mixer
        self.feed_forward = feed_forward
        self.norms = dict(norms)
        self.params = dict(params or {})
        self.token_input = token_input

    @classmethod
    def expected_tensors(cls, layer) -> list:
        """Tensors of the arrangement itself (not of its parts), by full name; ``layer``: the ``LayerSpec``."""
        return []

    def load(self, tensors: dict, layer, device, dtype) -> None:
        """Take the arrangement's own tensors."""

    def state_spec(self):
        """State the arrangement itself keeps per live request (None, a ``StateSpec`` or a dict of them);
        ``cache.block_state`` holds it."""
        return None

    def forward(self, ctx, acc, cache) -> None:
        raise NotImplementedError


class _Registry:
    def __init__(self, what: str):
        self.what = what
        self._items: dict[str, type] = {}

    def register(self, name: str) -> Callable[[type], type]:
        def _do(cls: type) -> type:
            cls.kind = name
            self._items[name] = cls
            return cls

        return _do

    def get(self, name: str) -> type:
        try:
            return self._items[name]
        except KeyError:
            raise KeyError(
                f"unknown {self.what} {name!r}; registered: {', '.join(sorted(self._items)) or 'none'}"
            ) from None

    def names(self) -> list[str]:
        return sorted(self._items)


MIXERS = _Registry("mixer")
FEED_FORWARDS = _Registry("feed-forward")
NORMS = _Registry("norm")
POSITIONS = _Registry("position encoding")
BLOCKS = _Registry("block arrangement")
TOKEN_INPUTS = _Registry("token input")


def build_part(registry: _Registry, spec: PartSpec) -> Part:
    return registry.get(spec.kind)(spec)
