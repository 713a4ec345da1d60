"""Interfaces of the parts a layer is put together from, and their registries.

A *part* is built from a ``PartSpec`` (kind + constants) alone; it never sees
the model configuration or knows which model it is in.  Five kinds exist:

``Norm``              y = f(x); optionally fused with the residual sum.
``PositionEncoding``  acts on the q and k heads of the step's tokens.
``Mixer``             mixes information across a request's tokens and owns
                      per-request memory through the cache manager (pages of
                      keys and values, or a record of fixed size).
``FeedForward``       acts on each token alone (dense or routed).
``Block``             the arrangement of the four above in a layer.

All parts declare their checkpoint tensors (``tensors``) with names relative to
their prefix, and receive them in ``load``.  Adding a part is: subclass,
``register_part("mixer", "my_kind", MyMixer)``, and name ``my_kind`` in a
``PartSpec`` of some architecture's ``model_spec``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Dict, List, Mapping, NamedTuple, Optional, Sequence, Tuple, Type

import torch

from ..config.spec import PartSpec


# --------------------------------------------------------------------------
# declarations
# --------------------------------------------------------------------------

@dataclass(frozen=True)
class TensorDecl:
    """A checkpoint tensor a part reads.

    ``role`` decides how it is kept on the device and how random weights are
    drawn: ``matrix`` (compute dtype, N(0, s_matrix)), ``bias`` (float32,
    N(0, s_bias)), ``norm`` (float32, 1 + N(0, s_norm)), ``table`` (int32).
    ``std`` replaces the role's standard deviation for this tensor (a mean of
    ``mean``), for tensors whose useful range is not the role's.
    A size given as None is one that only the checkpoint knows (the inner
    width of a low-rank pair, say): any size fits, the part reads it off the
    tensor in ``load``, and random weights cannot be drawn for it.
    """

    shape: Tuple[Optional[int], ...]
    role: str = "matrix"
    optional: bool = False
    std: Optional[float] = None
    mean: float = 0.0
    eye: float = 0.0               # random weights: this much of the identity is added (square matrices)
    # random weights: the shape to draw when ``shape`` has a size that only the checkpoint knows
    random_shape: Optional[Tuple[int, ...]] = None


@dataclass(frozen=True)
class PagedKVNeed:
    """Per-token memory in pages: a key plane and a value plane.  Planes with equal needs share a cache group.

    The two planes may have different widths (``value_head_dim``; None: as wide as the keys), and a mixer
    that keeps one vector per token only (a latent that serves as key and value) asks for
    ``value_head_dim=0``: its group then has no value plane at all.
    """

    num_kv_heads: int
    head_dim: int                          # width of a key
    window: Optional[int] = None           # None: every earlier position stays readable
    value_head_dim: Optional[int] = None   # width of a value; None: head_dim; 0: no value plane
    # a token reads the positions of its own chunk only (chunks of this many positions, counted from 0)
    chunk: Optional[int] = None
    # with a window: the request's first positions stay readable whatever the window (their pages are kept)
    keep_first: int = 0


@dataclass(frozen=True)
class StateNeed:
    """A record of fixed size per request (zeroed when the request slot is opened)."""

    shape: Tuple[int, ...]
    dtype: str = "float32"         # "float32", "bfloat16" or "compute" (the engine's dtype)


class Part:
    kind_family = ""

    def __init__(self, spec: PartSpec):
        self.spec = spec
        self.prefix = spec.prefix

    def tensors(self) -> Dict[str, TensorDecl]:
        """Checkpoint tensors of this part, names relative to ``self.prefix``."""
        return {}

    def load(self, fetch: Callable[[str], Optional[torch.Tensor]], dtype: torch.dtype, device: torch.device) -> None:
        """Take the tensors (``fetch(relative_name)`` gives a CPU tensor or None) onto the device."""

    def kernel_libraries(self) -> Sequence[str]:
        """Kernel libraries this part launches from (compiled before the first step)."""
        return ("core",)


class Norm(Part):
    kind_family = "norm"

    def split_params(self) -> Optional[Tuple[torch.Tensor, float]]:
        """(weight float32 [hidden], eps) if the norm is y = x / sqrt(mean(x^2) + eps) * weight, so that the
        products around it may split it between them (``NormSplit``); None otherwise."""
        return None

    def forward(self, x: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        raise NotImplementedError

    def add_forward(self, residual: torch.Tensor, delta: Optional[torch.Tensor],
                    rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """residual += delta (in place, unless ``rows`` selects rows), then the norm of it.

        The default is the unfused form; a part with a fused kernel overrides it.
        ``delta`` may also be float32 partial sums [parts, tokens, hidden] of a product that was
        split over its inner dimension; they are added up first.  A block whose parts all read one
        norm's output hands their outputs on as a tuple; they are added to each other first, then
        to the residual.
        """
        if isinstance(delta, ResidualCopy):
            delta = None
        delta = settled(delta, residual.dtype)
        if isinstance(delta, (tuple, list)):
            parts = [whole_output(d, residual.dtype).float() for d in delta if d is not None]
            delta = None
            if parts:
                delta = parts[0]
                for d in parts[1:]:
                    delta = delta + d
        if delta is not None and delta.dim() == 3:
            delta = delta.sum(0).to(residual.dtype)
        if rows is not None:
            picked = residual.index_select(0, rows.long())
            if delta is not None:
                picked = (picked.float() + delta.index_select(0, rows.long()).float()).to(residual.dtype)
            return self.forward(picked)
        if delta is not None:
            residual.copy_((residual.float() + delta.float()).to(residual.dtype))
        return self.forward(residual)


class PositionEncoding(Part):
    kind_family = "position"
    # True if `fused_table()` gives a cos/sin table that the fused
    # bias+rotation+store kernel understands (half-split pairs).
    fuses_with_store = False

    def apply(self, qkv: torch.Tensor, positions: torch.Tensor, num_heads: int, num_kv_heads: int,
              head_dim: int, num_tokens: int) -> None:
        """Encode positions into the q and k heads of ``qkv`` [tokens, (nh+2nkv)*hd], in place."""
        raise NotImplementedError

    def prepare(self, device: torch.device) -> None:
        """Build device tables (called once after ``load``)."""


class StepView:
    """What a part may know about the step that is running (``engine/batch.py`` fills it in).

    On the device, valid in every step, captured in a CUDA graph or not (int32 tensors):
      ``token_ids [tokens]``, ``positions [tokens]`` (place of each token in its request),
      ``token_req [tokens]`` (entry of each token), ``cu_q [entries + 1]`` (first token of each entry),
      ``ctx_len [entries]`` (tokens of the request cached before this step), ``req_slot [entries]``
      (the request's slot: the row of its block table and of its state record; -1 marks a padding entry,
      which a part skips or gives a defined output), ``status [1]`` (error word).
    On the host: ``num_tokens``, ``num_entries`` (padding included), ``num_single`` (the leading entries
    that bring exactly one token: single-token entries always come first), ``max_kv_len``, ``scratch`` (a
    dict that lives as long as the step, for plans shared by all layers).
    Only in steps that are not captured: ``entries`` (the host's list of entries, with their tokens) and
    ``entry_ctx``.  A step made of single-token entries only may be captured once and replayed with other
    contents of the device arrays: then ``captured`` is true, the arrays are padded to the bucket's size,
    and whatever a part does must depend on the device arrays alone: no host list, no ``.item()``, no
    shape that depends on the step's contents.  A portion of several tokens is never captured.
    """


class NormEntry(NamedTuple):
    """What the product before a norm has to know to prepare the norm's input for the part after the norm
    (``NormSplit``): the norm's weight and eps, and whether that part takes such an input for rows shaped like the
    residual rows it is asked about."""
    weight: torch.Tensor                          # float32 [hidden]
    eps: float
    accepts: Callable[[torch.Tensor], bool]


class NormSplit(NamedTuple):
    """A norm's input as the product before the norm left it, for the product after the norm: the residual rows
    (already summed and written back) times the norm's weight, and the rows' sums of squares in parts.  The product
    after the norm multiplies ``scaled`` and scales each row of its result by 1 / sqrt(sum / width + eps), so the
    norm needs no kernel of its own between two products of a decode step."""
    scaled: torch.Tensor      # [tokens, hidden], the engine's dtype
    sumsq: torch.Tensor       # float32 [parts, 32]: sums of squares of the rows' values, a part per 16 columns
    eps: float


class StreamWrite(NamedTuple):
    """A sublayer's output that has not been written into a residual of several streams yet (``parts/streams.py``):
    X[t] <- sum_s mix[s, t] X[s] + write[t] * y.  The norm that reads the residual next applies it in its pass."""
    y: torch.Tensor           # [tokens, hidden] in the engine's dtype, or float32 partial sums [parts, tokens, hidden]
    mix: torch.Tensor         # float32 [streams, streams]: row = the stream read, column = the stream written
    write: torch.Tensor       # float32 [streams]


class ResidualCopy(NamedTuple):
    """Handed on by a block in the place of a pending output when nothing is pending: the float32 residual rows,
    already summed, rounded to the engine's dtype (what the next block's products read, made in the pass that
    wrote the residual).  A norm that is given one has nothing to add."""
    rows: torch.Tensor        # [tokens, hidden] in the engine's dtype


class Pending(NamedTuple):
    """What has not been added to the residual yet, where it is more than one tensor: a sublayer's output ``y``, rows
    times a number a token (``rows``, ``rows_w``: experts that pass their input on), and float32 rows (``extra``: the
    embedding's output, which a layer range that runs again starts with).  A norm that reads a float32 residual adds
    them all in its pass; ``settled`` makes one tensor of them for the others."""
    y: Optional[torch.Tensor] = None         # [tokens, hidden], or float32 partial sums [parts, tokens, hidden]
    rows: Optional[torch.Tensor] = None      # [tokens, hidden] in the engine's dtype
    rows_w: Optional[torch.Tensor] = None    # float32 [tokens]
    extra: Optional[torch.Tensor] = None     # float32 [tokens, hidden]


class NormedOutput(NamedTuple):
    """A sublayer's output whose own norm is still to be taken: y / sqrt(mean(y^2) + eps) * weight (+ ``row``, one float32
    row for all tokens) is what the residual gains.  The norm that reads the residual next takes it in its pass."""
    y: Optional[torch.Tensor]                # [tokens, hidden], or float32 partial sums [parts, tokens, hidden]; None: the row alone
    weight: Optional[torch.Tensor] = None    # float32 [hidden]
    eps: float = 0.0
    row: Optional[torch.Tensor] = None       # float32 [hidden]

    def gain(self) -> Optional[torch.Tensor]:
        """What it adds to the residual, as float32 rows (for readers without a fused pass)."""
        if self.y is None:
            return None if self.row is None else self.row[None, :]
        y = self.y.sum(0) if self.y.dim() == 3 else self.y.float()
        out = y * torch.rsqrt((y * y).mean(-1, keepdim=True) + self.eps) * self.weight
        return out if self.row is None else out + self.row


def with_row(delta, row: torch.Tensor, tokens: int):
    """The pending output ``delta`` and one float32 ``row`` [hidden] for every token besides."""
    if delta is None or isinstance(delta, ResidualCopy):
        return NormedOutput(None, row=row)
    if isinstance(delta, NormedOutput):
        return delta._replace(row=row if delta.row is None else delta.row + row)
    return with_extra(delta, row[None, :].expand(tokens, -1).contiguous())


def with_extra(delta, extra: torch.Tensor) -> Pending:
    """The pending output ``delta`` and ``extra`` rows besides."""
    if delta is None or isinstance(delta, ResidualCopy):
        return Pending(extra=extra)
    if isinstance(delta, Pending):
        return delta._replace(extra=extra if delta.extra is None else delta.extra + extra)
    if isinstance(delta, NormedOutput):
        gain = delta.gain()
        return Pending(extra=extra if gain is None else extra + gain)
    if isinstance(delta, torch.Tensor):
        return Pending(y=delta, extra=extra)
    raise TypeError(f"rows cannot be added to a pending {type(delta).__name__}")


def settled(delta, dtype: torch.dtype):
    """A ``Pending`` (or a ``NormedOutput``) as one tensor of ``dtype`` (None if nothing is pending); anything else as it is."""
    if isinstance(delta, NormedOutput):
        gain = delta.gain()
        return None if gain is None else gain.to(dtype)
    if not isinstance(delta, Pending):
        return delta
    total = None if delta.y is None else (delta.y.sum(0) if delta.y.dim() == 3 else delta.y.float())
    if delta.rows is not None:
        part = delta.rows.float() * delta.rows_w[:, None]
        total = part if total is None else total + part
    if delta.extra is not None:
        total = delta.extra if total is None else total + delta.extra
    return None if total is None else total.to(dtype)


class Connection(Part):
    """How a sublayer is joined to the residual: what it reads (``read``: float32 weights over the streams) and how
    its output goes back (``write(y)`` gives the pending ``StreamWrite``)."""

    kind_family = "connection"
    read: Optional[torch.Tensor] = None

    def write(self, y) -> "StreamWrite":
        raise NotImplementedError


class Mixer(Part):
    kind_family = "mixer"

    def cache_need(self):
        """``PagedKVNeed``, ``StateNeed`` or None."""
        return None

    def sub_mixers(self) -> List[Tuple[str, "Mixer"]]:
        """The mixers a composite mixer is made of, with their names (empty for an ordinary mixer).  Each gets a
        cache plane of its own; the composite's ``forward`` is then given a dict name -> cache view."""
        return []

    # False: ``forward`` must return one [tokens, hidden] tensor, not partial sums (set by a composite on its members)
    partial_ok = True

    def prepare(self, device: torch.device, dtype: torch.dtype) -> None:
        pass

    # True: ``forward`` takes ``residual=h`` and may add its output to the residual stream itself (in its
    # last product's epilogue), returning None instead of the output
    accumulates = False
    # True: ``forward`` also takes ``into_norm=NormEntry`` (the norm after this part and what comes after it) and
    # may, for steps where that pays and the part after the norm accepts it, add its output to the residual stream
    # and return a ``NormSplit`` instead
    splits_norm = False

    def forward(self, x: torch.Tensor, step: "StepView", cache: Any) -> torch.Tensor:
        """x [tokens, hidden] -> [tokens, hidden].  ``cache`` is the view of this run-step's plane.

        The result may also be float32 partial sums [parts, tokens, hidden] of a last product that was
        split over its inner dimension: ``Norm.add_forward`` adds them up with the residual; a block that
        does anything else with the result passes it through ``whole_output`` first."""
        raise NotImplementedError


def whole_output(out: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
    """A part's output as one [tokens, hidden] tensor of ``dtype`` (partial sums added up)."""
    out = settled(out, dtype)
    if out.dim() == 3:
        return out.sum(0).to(dtype)
    return out


class FeedForward(Part):
    kind_family = "feed_forward"
    accumulates = False   # as for a mixer
    # True: ``forward`` accepts a ``NormSplit`` in place of the normalised rows where ``accepts_norm_split`` says so
    takes_norm_split = False

    def accepts_norm_split(self, rows: torch.Tensor) -> bool:
        """Whether a ``NormSplit`` may stand for normalised rows shaped like ``rows`` (the residual rows) in this step."""
        return False

    def forward(self, x: torch.Tensor, step: "StepView") -> torch.Tensor:
        raise NotImplementedError


class Block(Part):
    """An arrangement of parts in a layer.

    ``roles`` names the parts a block kind is made of and the family each is built from; the layer's
    ``LayerSpec.parts`` gives a ``PartSpec`` for every role.  Every built part is also an attribute of the
    block under its role's name.  ``forward`` gets the residual stream ``h``, a pending ``delta`` that has not
    been added to it yet (so that the sum can be fused into the next norm), and ``caches``: for every role
    of the mixer family, the view of that mixer's cache plane in this run-step (None if it keeps nothing).
    It returns ``(h, delta)`` again.
    """

    kind_family = "block"
    # True: ``forward`` never writes into the residual rows it is given (it returns other ones)
    keeps_residual = False
    roles: Mapping[str, str] = {}      # role -> family ("mixer", "feed_forward", "norm")

    def __init__(self, parts: Mapping[str, Part]):
        self.named: Dict[str, Part] = dict(parts)
        for role, part in self.named.items():
            setattr(self, role, part)

    def parts(self) -> List[Part]:
        return [self.named[role] for role in self.roles]

    def mixers(self) -> List[Tuple[str, "Mixer"]]:
        """The block's mixers with their roles, in the order of ``roles``."""
        return [(role, self.named[role]) for role, family in self.roles.items() if family == "mixer"]

    def cache_users(self) -> List[Tuple[str, "Mixer"]]:
        """Every mixer that may own memory in the cache manager, by path: ``role`` for an ordinary mixer,
        ``role.name`` for the members of a composite one."""
        out: List[Tuple[str, "Mixer"]] = []

        def walk(path: str, m: "Mixer") -> None:
            subs = m.sub_mixers()
            if not subs:
                out.append((path, m))
            for name, sub in subs:
                walk(f"{path}.{name}", sub)

        for role, m in self.mixers():
            walk(role, m)
        return out

    def forward(self, h: torch.Tensor, delta: Optional[torch.Tensor], step: "StepView", caches: Mapping[str, Any]):
        raise NotImplementedError


# --------------------------------------------------------------------------
# registries
# --------------------------------------------------------------------------

_REGISTRY: Dict[str, Dict[str, Any]] = {
    "norm": {}, "position": {}, "mixer": {}, "feed_forward": {}, "block": {}, "embedding": {}, "head": {},
    "connection": {},
}


def register_part(family: str, kind: str, cls: Any) -> None:
    if family not in _REGISTRY:
        raise KeyError(f"unknown part family {family!r}; families: {sorted(_REGISTRY)}")
    _REGISTRY[family][kind] = cls


def part_class(family: str, kind: str):
    try:
        return _REGISTRY[family][kind]
    except KeyError:
        raise KeyError(
            f"no {family} part of kind {kind!r} is registered; known: {sorted(_REGISTRY.get(family, {}))}"
        ) from None


def build_part(family: str, spec: PartSpec):
    return part_class(family, spec.kind)(spec)
