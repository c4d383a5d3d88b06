"""Interfaces of the parts a layer is put together from, and one registry per kind of part.

A part is built from the parameters of its :class:`~transformer_b200.parts.spec.PartSpec` alone; it
does not know which model it is in, which layer it is, or what the other parts are.  The engine
talks to parts only through the methods below.

============  ===================================================================================
kind          interface
============  ===================================================================================
Embedding     ``forward(ctx, x)``: fill the float residual stream ``x`` [nt, d] for the step's tokens
              (``ctx.tok_ids``, and ``ctx.tok_pos`` for an encoding that adds positions here).  With a
              ``state_need()`` it is handed its per-sequence state as ``state=``.
Norm          ``forward(ctx, x, delta, rows, y)``: ``v = x[rows] + delta[rows]`` (float sum; written
              back to ``x`` when ``rows`` is None), ``y = norm(v)``.  ``x`` is the float residual
              stream, ``delta`` the previous part's output or None.
Mixer         ``forward(ctx, x1, out, cache, state)``: reads the normed activations ``x1`` [nt, d]
              and writes its contribution to the stream into ``out`` [nt, d].  ``cache`` is what the
              storage class of its ``cache_need().kind`` shows a run (None if ``cache_need()`` is
              None), ``state`` its per-sequence state tensor [slots, *shape] (None if
              ``state_need()`` is None); rows of ``state`` are addressed by ``ctx.slots``.
FeedForward   ``forward(ctx, x1, out)``; may return a ``WeightedRows`` instead of filling ``out``.
Position      owned by the mixer that uses it.  A rotary encoding answers ``rotation()`` with its
              (cos, sin, half_pairing) and the mixer fuses the rotation with its cache write; any
              other encoding answers None and is called as ``apply(ctx, qkv, nh, nkvh, dh)`` to
              change the step's queries and keys in place by its own means.
Head          ``forward(ctx, xn, logits)``: float logits [rows, vocab] of the normed rows ``xn``.
Arrangement   how a layer's parts are put together in a block: built from a LayerSpec,
              ``parts()`` (name -> part), ``mixer``, ``forward(ctx, x, pending, cache, state)``.  An
              arrangement whose parts other than the mixer carry state per sequence offers ``state_needs()``
              (name -> StateNeed) and is handed ``state`` as a dict of the same names.
InputFilter   changes what a part reads, row by row or along time: ``forward(ctx, y, out, state)`` with
              ``y`` the normed rows [nt, d]; it may carry per-sequence state (``state_need()``).
Joint         rewrites the whole residual stream between two runs of the model: ``begin(ctx, x)`` right after
              the embedding (to keep what it needs of it), ``forward(ctx, x, pending)`` before the run that
              names it (``pending`` is what the run before left to be added; it returns what is still pending).
ResidualGate  multiplies a part's result before it joins the stream, by a function of what that part reads:
              ``forward(ctx, y)`` gives the gate's pre-activation [nt, d] and its bias; the sum applies them.
============  ===================================================================================

All parts declare their parameters with :meth:`Part.parameters` (name -> shape, role, init) and
receive the device tensors with :meth:`Part.bind`.  A part whose ``forward`` only launches work on the
device that reads the step's numbers from ``ctx``'s DEVICE arrays (never from the ``h_*`` host lists,
never a value copied back to the host) may set ``graph_safe = True``: decode steps of a model whose
parts all say so are captured into CUDA graphs and replayed with new index arrays.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Dict, Optional, Tuple

import torch


@dataclass(frozen=True)
class ParamDecl:
    shape: Tuple[int, ...]
    role: str = "matrix"     # "matrix" | "norm" | "table"
    init: str = "normal"     # "normal" | "ones" | "distinct:n" (a table: integers below n, those of a row differing)


@dataclass(frozen=True)
class CacheNeed:
    """What a mixer wants kept for every sequence: ``kind`` names a registered storage class
    (:data:`transformer_b200.cache.paged.CACHE_KINDS`; "full" = keys and values of every position in pages),
    for nkvh heads of size dh; ``params`` holds what else the kind needs (a window's length, ...).  Runs with
    equal needs share one storage object."""
    kind: str
    nkvh: int
    dh: int
    params: Tuple[Tuple[str, Any], ...] = ()

    def get(self) -> Dict[str, Any]:
        return dict(self.params)


@dataclass(frozen=True)
class StateNeed:
    """A tensor of fixed size per sequence, zero when a sequence starts."""
    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass
class WeightedRows:
    """A part's output that is not summed yet: out[t] = sum_j weights[t, j] * rows[index[t * k + j]].
    A norm that sets ``takes_weighted_rows`` does the sum itself, in float, while it adds to the stream
    (one kernel and one round trip through memory less); for any other norm the block sums first."""
    rows: torch.Tensor        # [M, d]
    index: torch.Tensor       # int32 [nt * k]
    weights: torch.Tensor     # float [nt, k]
    k: int


@dataclass
class PairDelta:
    """Two parts' outputs that are still to be added to the stream together:  x += (first + second), summed in
    float.  Left by a block whose mixer and feed-forward read the same stream.  A norm that sets
    ``takes_pair_delta`` does the sum in its own kernel; for any other the block adds it to the stream first."""
    first: torch.Tensor       # [nt, d]
    second: Optional[torch.Tensor]


@dataclass
class NormedDelta:
    """A part's output that still has to be normed before it joins the stream:  x += delta / rms(delta) * weight
    (a block that norms its parts' outputs as well as their inputs).  ``delta`` is a tensor [nt, d] or a
    :class:`WeightedRows`.  A norm that sets ``takes_normed_delta`` does that norm, the sum and its own norm in one
    kernel; for any other norm the block applies it to the stream first (:func:`parts.block.resolve`).
    With ``center`` the norm is a layer norm: x += (delta - mean) / sqrt(var(delta) + eps) * weight + bias."""
    delta: Any
    weight: torch.Tensor      # float [d]
    eps: float
    bias: Optional[torch.Tensor] = None     # float [d]
    center: bool = False


@dataclass
class GatedDelta:
    """A part's output that passes a bias and a gate of its own on its way into the stream, element by element:
    x += (delta + delta_bias) * sigmoid(gate + gate_bias); each of the three but ``delta`` may be missing.  A norm that
    sets ``takes_gated_delta`` does the sum in its own kernel; for any other the block adds it to the stream first."""
    delta: torch.Tensor                            # [nt, d]
    delta_bias: Optional[torch.Tensor] = None      # float [d]
    gate: Optional[torch.Tensor] = None            # [nt, d]
    gate_bias: Optional[torch.Tensor] = None       # float [d]

    def moved(self, of: Callable) -> "GatedDelta":
        """The same left by another run of an equal layer: ``of`` maps a layer's own tensor to the other layer's."""
        return GatedDelta(self.delta, of(self.delta_bias), self.gate, of(self.gate_bias))


@dataclass
class DepthSum:
    """The stream is still to be replaced by a weighted sum over the depth of the model: with ``pending`` added first,
    X = x (which is kept as the last of ``terms`` rows of ``history``), x <- sum_j weights[j] history[j].  Norms with
    ``takes_gated_delta`` do all of it in their own kernel."""
    pending: Any               # a tensor, a GatedDelta or None
    history: torch.Tensor      # float [>= terms, nt, d]; the first terms - 1 are filled
    weights: torch.Tensor      # float [terms]
    terms: int


@dataclass
class StreamRows:
    """Nothing is left to be added to the stream, and the stream's rows, rounded to the activation type, already lie in
    ``rows``: left by a block whose last kernel norms the stream itself, for a block that reads it as it is."""
    rows: torch.Tensor        # [nt, d]


class Part:
    graph_safe = False      # see the head of this file; the parts of this package set it
    launches_only = False   # all device work goes through csrc.lib launchers (or reports itself with lib.foreign):
                            # the engine may then record one layer's launches and replay them for its equals

    def __init__(self, params: Dict[str, Any], dtype: torch.dtype, device: torch.device):
        self.params = dict(params)
        self.dtype = dtype
        self.device = device
        self.weights: Dict[str, torch.Tensor] = {}

    def parameters(self) -> Dict[str, ParamDecl]:
        return {}

    def early_weights(self) -> Optional[torch.Tensor]:
        """A small weight that this part reads first and waits for (a router's matrix), or None.  The part that
        runs before it may ask for it to be brought into L2 meanwhile (``Norm.forward(..., warm=)``)."""
        return None

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        decl = self.parameters()
        for name, d in decl.items():
            t = tensors[name]
            if tuple(t.shape) != tuple(d.shape):
                raise ValueError(f"{type(self).__name__}.{name}: shape {tuple(t.shape)}, expected {d.shape}")
        self.weights = {n: tensors[n] for n in decl}


@dataclass
class NormTail:
    """A small computation on the rows a norm has just produced, which the part after the norm asks it to do in
    the same kernel (the rows are at hand there; a kernel of its own would wait for them and read them back).
    ``kind`` names it; a norm lists the kinds it can do in ``Norm.tails`` and is handed nothing else.
    "router": ``weights`` [E, d], ``k``; the norm fills ``index`` [rows, k] (int32) and ``scores`` [rows, k] (float)
    with each row's k experts and their softmax weights, by the rules of the router kernel.
    "terms": the experts that ``table`` gives the row's token, and what ``gate`` gives an expert besides."""
    kind: str
    weights: Any = None
    k: int = 0
    index: Any = None
    scores: Any = None
    scored: bool = False     # "router": softmax over all outputs, choice by score + bias, weights = the chosen scores
    bias: Any = None
    sigmoid: bool = False    # "router": the k largest logits, weights = their sigmoids as they are
    table: Any = None        # "terms": [vocab, k] int32, the experts of every token id, each with weight 1 / k
    gate: Any = None         # "terms": [d], the gate of an expert that every token passes; ``scores`` is then [rows, k + 1],
                             #          the last entry sigmoid(gate . row)

    @property
    def rule(self) -> int:
        """The kernels' number of the rule of choice (csrc/router_pick.cuh)."""
        return 2 if self.sigmoid else 1 if self.scored else 0


class Norm(Part):
    takes_weighted_rows = False
    takes_normed_delta = False
    takes_pair_delta = False
    takes_gated_delta = False  # a GatedDelta or a DepthSum
    can_warm = False           # forward takes ``warm=``: a weight of the next part to fetch into L2 meanwhile
    tails: tuple = ()          # kinds of NormTail that forward(..., tail=) computes along the way
    renew_tails: tuple = ()    # the same for renew(..., tail=)

    def forward(self, ctx, x, delta, rows, y) -> None:
        raise NotImplementedError

    def renew(self, ctx, x, delta, y, tail=None) -> None:
        """x <- y = norm(stream * x + delta), x in float, y rounded to the activation type; ``stream`` is the norm's own
        parameter.  For blocks that norm the stream itself (optional)."""
        raise NotImplementedError


class Mixer(Part):
    rows_width: Optional[int] = None    # the width of the rows that forward_rows leaves for the output product
    in_weight: Optional[str] = None     # name of the weight [in_width, width] of a first product z = x1 weight^T that whoever
    in_width: int = 0                   # calls the mixer may do together with others that read x1: ``forward`` and
                                        # ``forward_rows`` then take the rows (a view with a pitch) as ``z=``
    has_out_bias = False                # ``out_bias``, float [d], is still to be added to what forward writes: the block
    out_bias: Optional[torch.Tensor] = None      # does that where it adds the result to the stream (``takes_out_bias``)

    def cache_need(self) -> Optional[CacheNeed]:
        return None

    def state_need(self) -> Optional[StateNeed]:
        return None

    def forward(self, ctx, x1, out, cache, state) -> None:
        raise NotImplementedError

    def forward_rows(self, ctx, x1, rows, cache, state) -> None:
        """What ``forward`` does up to its output product (weight "wo", [width, rows_width]): ``rows`` [nt, rows_width],
        a view with a pitch, receives what that product reads.  For mixers that stand beside another one."""
        raise NotImplementedError


class FeedForward(Part):
    def norm_tail(self, ctx, nt: int) -> Optional[NormTail]:
        """What the norm before this part may compute along the way in a step of ``nt`` rows, or None.  If the norm
        lists the kind, it is handed the object and ``forward`` receives it back as ``tail=`` (computed)."""
        return None

    def forward(self, ctx, x1, out):
        """Write the contribution into ``out`` and return None, or return a :class:`WeightedRows`
        that stands for it (``out`` is then left alone)."""
        raise NotImplementedError


class InputFilter(Part):
    def state_need(self) -> Optional[StateNeed]:
        return None

    def forward(self, ctx, y, out, state) -> None:
        raise NotImplementedError


class Joint(Part):
    def begin(self, ctx, x) -> None:
        """Called once per step with the embedding output ``x`` (float [nt, d]), before any layer runs."""

    def forward(self, ctx, x, pending):
        raise NotImplementedError


class ResidualGate(Part):
    product: Optional[str] = None       # name of the weight [d, width] if the pre-activation is y weight^T: the block may
                                        # do that product together with another one and hand its rows over as ``z=``

    def forward(self, ctx, y, z=None) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
        """The gate's pre-activation for the rows ``y`` that the gated part reads, and a bias to be added to it."""
        raise NotImplementedError


class Position(Part):
    def rotation(self):
        """(cos, sin, half_pairing) of a rotary encoding -- float tables [positions, dh/2] on the device and 0
        for adjacent pairs (2i, 2i+1), 1 for halves (i, i + dh/2) -- or None for any other encoding."""
        return None

    def apply(self, ctx, qkv, nh: int, nkvh: int, dh: int) -> None:
        """For an encoding without ``rotation()``: change the step's queries and keys in place.  ``qkv`` is
        [nt, (nh + 2 nkvh) dh] with the heads in the order q, k, v; ``ctx.tok_pos`` holds the positions."""
        raise NotImplementedError


class Embedding(Part):
    def state_need(self) -> Optional[StateNeed]:
        """A tensor of fixed size per sequence that the embedding carries from step to step (the token before, for
        an embedding of token pairs), or None.  An embedding that asks for one is called as
        ``forward(ctx, x, state=)`` with the tensor [slots, *shape]; rows are addressed by ``ctx.slots``."""
        return None

    def forward(self, ctx, x) -> None:
        raise NotImplementedError


class Head(Part):
    def forward(self, ctx, xn, logits) -> None:
        raise NotImplementedError


class Registry:
    def __init__(self, what: str):
        self.what = what
        self._kinds: Dict[str, Callable] = {}

    def register(self, kind: str, cls=None, *, replace: bool = False):
        def deco(c):
            if kind in self._kinds and not replace:
                raise ValueError(f"{self.what} kind {kind!r} is already registered")
            self._kinds[kind] = c
            return c
        return deco(cls) if cls is not None else deco

    def unregister(self, kind: str) -> None:
        self._kinds.pop(kind, None)

    def get(self, kind: str):
        cls = self._kinds.get(kind)
        if cls is None:
            raise ValueError(f"unknown {self.what} kind {kind!r}; registered: {sorted(self._kinds)}")
        return cls

    def build(self, spec, dtype, device):
        return self.get(spec.kind)(spec.get(), dtype, device)

    def kinds(self):
        return sorted(self._kinds)


EMBEDDINGS = Registry("embedding")
HEADS = Registry("head")
NORMS = Registry("norm")
MIXERS = Registry("mixer")
FEED_FORWARDS = Registry("feed-forward")
POSITIONS = Registry("position encoding")
INPUT_FILTERS = Registry("input filter")
JOINTS = Registry("joint")
RESIDUAL_GATES = Registry("residual gate")
ARRANGEMENTS = Registry("block arrangement")     # kind -> class(LayerSpec, dtype, device); see parts/block.py
