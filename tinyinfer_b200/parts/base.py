"""Interfaces of the parts a decoder block is made of, and the registries that map a spec's
``kind`` to the class that runs it.

A part gets its sizes and constants from its spec, declares the tensors it wants by local name,
and is handed, at every step, the batch (``StepContext``) and, for mixers, a view of the cache
entry it works on. It never sees the model's configuration.

To add a part: write a spec dataclass with a ``kind`` field, a class deriving from ``Mixer``,
``FeedForward``, ``Norm`` or ``PositionEncoding``, and call the matching ``register_*``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Dict, Optional, Tuple

import torch


@dataclass(frozen=True)
class TensorSpec:
    """A tensor a part wants from the checkpoint.
    role 'matrix': kept in the compute dtype (bfloat16 or float32);
    role 'vector32': kept in float32 whatever the compute dtype (norm weights, biases of
    32-bit parts); role 'int': kept as int32 (random-weights mode: every row ``shape[-1]`` different numbers below ``below``). A size of -1 is one that only the checkpoint gives (the
    loader accepts any; the random-weights mode cannot draw such a tensor)."""
    shape: Tuple[int, ...]
    role: str = "matrix"
    init: str = "normal"          # random-weights mode: 'normal' N(0, std), 'ones_noise' 1 + N(0, 0.1) or
                                  # 'eye_noise' (a square matrix) identity + N(0, 0.1)
    below: int = 1


@dataclass(frozen=True)
class CacheNeed:
    """Paged keys and values a mixer wants per token: ``num_kv_heads * head_dim`` for K and V
    each. ``window`` None: every key stays; n: only the last n positions are ever read, older
    pages may be given back. ``chunk`` n: a position reads its own chunk of n positions only (chunks
    counted from position 0 of the request), so the pages of earlier chunks may be given back. ``keep_first`` n: beside the
    window the first n positions are read to the end of the request, so their pages stay."""
    num_kv_heads: int
    head_dim: int
    window: Optional[int] = None
    planes: int = 2          # 2: keys and values; 1: one row per token (a latent that both are made from)
    chunk: Optional[int] = None
    keep_first: int = 0

    @property
    def keeps_all(self) -> bool:
        """Every key stays to the end of its request."""
        return self.window is None and self.chunk is None

    def first_read(self, position: int) -> int:
        """The lowest position that a query at ``position`` or later reads (beside the ``keep_first`` first ones)."""
        if self.chunk is not None:
            return position // self.chunk * self.chunk
        return 0 if self.window is None else max(0, position - self.window + 1)


@dataclass(frozen=True)
class StateNeed:
    """Per-request state of fixed size (for instance a recurrent state): one slot of ``shape``
    per live request, zeroed when the request is admitted."""
    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


def state_slices(state: torch.Tensor, shapes):
    """Cuts a per-request state float32 [slots, n] into consecutive pieces of the given shapes:
    views [slots, *shape] whose slots lie as far apart as the whole state's."""
    out, at = [], 0
    for shape in shapes:
        n = 1
        for d in shape:
            n *= d
        out.append(state[:, at:at + n].unflatten(1, tuple(shape)))
        at += n
    if at > state.shape[1]:
        raise ValueError(f"a state of {state.shape[1]} floats a slot does not hold {at}")
    return out


class Part:
    def __init__(self, spec, dtype: torch.dtype, device):
        self.spec = spec
        self.dtype = dtype
        self.device = device

    def tensors(self) -> Dict[str, TensorSpec]:
        """Local tensor names (e.g. 'q_proj.weight') and what they must look like."""
        return {}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Receives exactly the tensors named by ``tensors()``, on the device, role applied."""

    def parts(self):
        """The parts this part is made of, if any (a mixer of several mixers): whoever lets go of a model's
        tensors walks through them."""
        return []


class Norm(Part):
    def forward(self, x: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError

    def forward_rows(self, x: torch.Tensor, rows: torch.Tensor) -> torch.Tensor:
        """Norm of the selected rows only. Parts without a fused kernel may gather first."""
        return self.forward(x.index_select(0, rows.long()))

    def as_rms(self):
        """(weight float32 [size], eps) if this norm is y = weight * x * rsqrt(mean(x^2) + eps), so
        that the products around it may share it between them (``ops.linear``); None otherwise."""
        return None


class PositionEncoding(Part):
    """Owned by a mixer, to which it hands ``rotation()``: an ``ops.Rotation`` (which features are paired,
    and each pair's angle at every position, as inverse frequencies or as a table of cosines and sines)
    or None if positions are not used. The mixer passes it to the fused norm + rotation + append kernel
    without looking inside. A part that sets ``inv_freq`` (float32 [rotary_dim / 2]) and ``rotary_dim``
    gets the half-split rotation by position * inv_freq from the default below."""
    inv_freq = None
    rotary_dim = 0

    def rotation(self):
        if self.inv_freq is None:
            return None
        from .. import ops
        return ops.Rotation(self.rotary_dim, inv_freq=self.inv_freq)


class Mixer(Part):
    # True if forward() only launches kernels on the step's device tensors (no host reads, no
    # Python branching on the step's contents): such a step may be captured in a CUDA graph.
    graph_safe = False

    def cache_need(self) -> Optional[CacheNeed]:
        return None

    def state_need(self) -> Optional[StateNeed]:
        return None

    def forward(self, x: torch.Tensor, step, cache) -> torch.Tensor:
        """x [T, hidden] (normed) -> [T, hidden]. ``step`` is the StepContext of the batch,
        ``cache`` the CacheView of the entry this run works on."""
        raise NotImplementedError

    def forward_residual(self, x, residual, step, cache) -> torch.Tensor:
        """residual + forward(x). Parts whose last kernel can add the residual override this."""
        from .. import ops
        return ops.add(residual, self.forward(x, step, cache))

    def forward_scaled(self, x, scale: float, residual, step, cache) -> torch.Tensor:
        """scale * forward(x) (+ residual): what a mixer that runs beside others contributes to their sum.
        Parts that can fold the factor into a kernel they launch anyway override this."""
        if scale != 1.0:
            raise NotImplementedError(f"{type(self).__name__} cannot scale its output; it cannot stand in a sum of mixers")
        return self.forward(x, step, cache) if residual is None else self.forward_residual(x, residual, step, cache)

    def input_rows(self):
        """(weight [n, hidden], bias float32 [n] or None) of the product that reads the mixer's input, if the mixer can
        take that product's result from someone else (``forward_projected``); None otherwise. A mixer of several
        mixers packs its branches' rows into one product. Once they are taken, the mixer's own copy may be dropped
        (``drop_input_rows``)."""
        return None

    def drop_input_rows(self) -> None:
        pass

    def forward_projected(self, projected, offset: int, x, scale: float, residual, step, cache) -> torch.Tensor:
        """``forward_scaled`` with the input product already made: its result for this mixer lies in columns
        [offset, offset + n) of ``projected``."""
        raise NotImplementedError

    def forward_prenorm(self, x, norm: "Norm", link, next_norm: Optional["Norm"], step, cache):
        """x + forward(norm(x)) for ``x`` BEFORE its norm. ``link``: None, or what the part that made x
        left for this norm (an ``ops.NormLink``); ``next_norm``: the norm the result will pass through
        next, if known. Returns (result, link for that next norm or None). Parts whose products can
        share a norm between them override this; the default runs the norm on its own."""
        return self.forward_residual(norm.forward(x), x, step, cache), None


class FeedForward(Part):
    def runs_beside(self, num_tokens: int) -> bool:
        """Whether a step of so many tokens gains from running this part beside a mixer that reads the same input (few tokens:
        chains of short kernels), and none of its kernels' CTAs wait for one another then (see ``ops.Beside``)."""
        return False

    graph_safe = False      # as for a mixer: a feed-forward that picks its experts' rows on the host is not

    def forward(self, x: torch.Tensor, step) -> torch.Tensor:
        raise NotImplementedError

    def forward_residual(self, x, residual, step) -> torch.Tensor:
        from .. import ops
        return ops.add(residual, self.forward(x, step))

    def forward_prenorm(self, x, norm: "Norm", link, next_norm: Optional["Norm"], step):
        """As ``Mixer.forward_prenorm``, without a cache."""
        return self.forward_residual(norm.forward(x), x, step), None


class Block:
    """An arrangement of one mixer, one feed-forward and their norms (``feed_forward`` and its norm are None in
    a block that has a mixer only; an arrangement that allows that says so in its own ``forward``)."""

    def __init__(self, spec, mixer: Mixer, feed_forward: FeedForward, mixer_norm: Norm,
                 feed_forward_norm: Norm):
        self.spec = spec
        self.mixer = mixer
        self.feed_forward = feed_forward
        self.mixer_norm = mixer_norm
        self.feed_forward_norm = feed_forward_norm

    def tensors(self) -> Dict[str, TensorSpec]:
        """Tensors the arrangement itself owns, named from the layer's prefix (most have none)."""
        return {}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        pass

    def state_need(self) -> Optional[StateNeed]:
        """Per-request state of the whole block: its mixer's, and what the arrangement keeps itself, if anything."""
        return self.mixer.state_need()

    def forward(self, x, step, cache):
        raise NotImplementedError

    def forward_linked(self, x, link, next_norm: Optional[Norm], step, cache):
        """``forward`` that also takes what the block before left for this block's first norm and
        returns what this block leaves for ``next_norm`` (the first norm behind it): (x, link)."""
        return self.forward(x, step, cache), None


# ------------------------------------------------------------------ registries
_MIXERS: Dict[str, Callable] = {}
_FEED_FORWARDS: Dict[str, Callable] = {}
_NORMS: Dict[str, Callable] = {}
_POSITIONS: Dict[str, Callable] = {}
_BLOCKS: Dict[str, Callable] = {}


def _register(table, what):
    def register(kind: str, factory: Callable) -> None:
        table[kind] = factory
    register.__doc__ = f"Registers the class that runs {what} specs of this kind."
    return register


def _build(table, what):
    def build(spec, *args, **kwargs):
        kind = getattr(spec, "kind", None)
        if kind not in table:
            raise KeyError(f"no {what} registered for kind {kind!r}; known: {sorted(table)}")
        return table[kind](spec, *args, **kwargs)
    return build


register_mixer = _register(_MIXERS, "mixer")
register_feed_forward = _register(_FEED_FORWARDS, "feed-forward")
register_norm = _register(_NORMS, "norm")
register_position = _register(_POSITIONS, "position-encoding")
register_block = _register(_BLOCKS, "block arrangement")
build_mixer = _build(_MIXERS, "mixer")
build_feed_forward = _build(_FEED_FORWARDS, "feed-forward")
build_norm = _build(_NORMS, "norm")
build_position = _build(_POSITIONS, "position-encoding")


def build_block(spec, dtype, device) -> Block:
    if spec.arrangement not in _BLOCKS:
        raise KeyError(f"no block arrangement {spec.arrangement!r}; known: {sorted(_BLOCKS)}")
    return _BLOCKS[spec.arrangement](
        spec,
        build_mixer(spec.mixer, dtype, device),
        build_feed_forward(spec.feed_forward, dtype, device) if spec.feed_forward is not None else None,
        build_norm(spec.mixer_norm, dtype, device),
        build_norm(spec.feed_forward_norm, dtype, device) if spec.feed_forward_norm is not None else None)
