"""Interfaces of the parts a model is put together from, and their registries.

A part knows its own sizes and constants (its ``params``), declares the tensors
it needs under its name prefix, and runs on packed tokens.  It does not know
which model it is in, which layer it is, or what the other parts are.  The five
kinds:

* ``Norm``             - ``forward(residual, branch, ctx, rows=None) -> x``: adds the pending
  branch output into the float32 residual stream and returns the normalised rows.
* ``Mixer``            - ``forward(x, ctx, cache) -> Branch``: mixes tokens of one sequence
  (attention here); may keep keys/values or fixed-size state per sequence.
* ``FeedForward``      - ``forward(x, ctx) -> Branch``: per-token transformation.

One optional refinement: a consumer that sets ``TAKES_ROW_SCALE`` gets ``row_scale=`` beside ``x``, and the norm
may then leave its division by the root mean square to the consumer's first product (``Norm.forward_unscaled``): a
product is linear in its rows.  A norm that does so needs no whole row in one place, so the few rows of a decode
step can be spread over many blocks that never wait for one another.
* ``PositionEncoding`` - gives mixers a rotation table and/or adds to the embeddings.
* ``Block``            - arranges norms, a mixer and a feed-forward around the residual stream.

The reference has one hard-wired arrangement (Inference/ForwardPass.cs:199-267);
its fused ops ``AddRmsNormResidual`` / ``AddRmsNorm`` (IComputeBackend.cs:417-438)
are the ``Norm.forward`` contract here.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Callable, Dict, Optional, Tuple

import torch


@dataclass(frozen=True)
class TensorDecl:
    """A tensor a part needs: its shape and what it is (decides random initialisation)."""

    shape: Tuple[int, ...]
    role: str = "matrix"       # "matrix" | "norm" | "bias" | "table" | "stream_gain" | "stream_mix" | "conv" | "rate"
    optional: bool = False


@dataclass(frozen=True)
class Term:
    """One summand of what enters the residual: float32 partials ``[S, N, H]``; with ``weight`` (float32 ``[H]``) their sum
    is divided by its own root mean square (``eps`` inside the root) and multiplied by that weight first; with ``gain``
    (float32 ``[H]``) it is multiplied by that vector element by element; ``scale`` times the result is added."""

    data: torch.Tensor
    weight: Optional[torch.Tensor] = None
    eps: float = 0.0
    scale: float = 1.0
    gain: Optional[torch.Tensor] = None


@dataclass
class Branch:
    """Output of a mixer or feed-forward that has not been added to the residual stream yet.

    ``data`` is ``[n_partials, n_tokens, hidden]``; the partials (split-K slices of a
    matrix product, in float32) are summed by whoever consumes the branch.  ``write``: for a residual that is
    more than one stream, the part that holds the weights with which this branch enters the streams (set by the
    block that arranged the sublayer; ``None`` where the branch is simply added).  ``more``: further sets of
    partials ``[s_i, n_tokens, hidden]`` that enter the residual together with ``data`` (sublayers that read the
    same norm's output side by side); ``scale``: the factor on the whole sum as it is added.  ``terms``: instead of all
    that, the summands one by one (``Term``), each with a norm and a factor of its own; ``data`` is then the first term's.
    ``bias`` (float32 ``[H]``): added to every token together with ``data`` (the bias of the sublayer's last projection).
    Only norms that say so take ``more``, a scale other than 1, terms or a bias (``Norm.check_plain`` is for the others).
    """

    data: torch.Tensor
    write: Any = None
    more: Tuple[torch.Tensor, ...] = ()
    scale: float = 1.0
    terms: Tuple[Term, ...] = ()
    bias: Optional[torch.Tensor] = None

    @property
    def n_partials(self) -> int:
        return self.data.shape[0]

    def with_gain(self, gain: torch.Tensor) -> "Branch":
        """The branch with every summand multiplied by ``gain`` (float32 ``[H]``) element by element."""
        if any(t.gain is not None for t in self.as_terms()):
            raise ValueError("a branch's summands have a gain already")
        return Branch.of_terms(replace(t, gain=gain) for t in self.as_terms())

    @classmethod
    def of_terms(cls, terms) -> "Branch":
        terms = tuple(terms)
        if not terms:
            raise ValueError("a branch needs at least one term")
        return cls(terms[0].data, terms=terms)

    def as_terms(self) -> Tuple[Term, ...]:
        """The branch as a list of summands, whichever way it was built (``write`` has no such reading)."""
        if self.write is not None:
            raise ValueError("a branch that enters the residual through a part of its own has no plain terms")
        if self.bias is not None:
            raise ValueError("a branch with a bias has no plain terms: only a norm that takes the bias can add it")
        if self.terms:
            return self.terms
        return tuple(Term(d, scale=self.scale) for d in (self.data,) + tuple(self.more))


@dataclass(frozen=True)
class KvNeed:
    """A mixer keeps keys and values per position: ``window`` = 0 for all of them; ``value_dim`` = 0 for value
    heads of the key heads' size; ``values_in_keys``: a position's value IS its key (or a leading part of it), so one
    set of pages serves as both (the view's ``v_pages`` is its ``k_pages``)."""

    num_kv_heads: int
    head_dim: int
    window: int = 0
    value_dim: int = 0
    values_in_keys: bool = False


@dataclass(frozen=True)
class StateNeed:
    """A mixer keeps a fixed-size state per sequence, zeroed when a sequence starts."""

    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class MultiNeed:
    """A part keeps several things per sequence: ``needs`` is ``((name, need), ...)`` with each need a ``KvNeed``, a
    ``StateNeed`` or another ``MultiNeed``.  The cache hands the part a ``MultiView`` whose ``[name]`` is the view of that
    need."""

    needs: Tuple[Tuple[str, Any], ...]

    @classmethod
    def of(cls, **needs) -> Optional["MultiNeed"]:
        kept = tuple((k, v) for k, v in needs.items() if v is not None)
        return cls(kept) if kept else None


class Part:
    """Base of all parts.  ``params`` holds every size and constant; ``prefix`` the tensor names."""

    def __init__(self, params: Dict[str, Any], prefix: str, env: "BuildEnv"):
        self.params = dict(params)
        self.prefix = prefix
        self.env = env

    def tensors(self) -> Dict[str, TensorDecl]:
        """Tensor name (relative to the prefix) -> declaration."""
        return {}

    def tensor_name(self, rel: str) -> str:
        """The name under which a checkpoint stores the tensor this part calls ``rel``: the prefix and ``rel``,
        or what the part's ``tensor_names`` parameter says instead of ``rel`` (checkpoints of other families
        name a norm's weight or a projection's matrix in their own way)."""
        return self.prefix + self.params.get("tensor_names", {}).get(rel, rel)

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Receive the loaded tensors (same relative names); fuse or re-lay-out here."""

    def cache_need(self):
        return None


def as_f32(t: torch.Tensor, env: "BuildEnv") -> torch.Tensor:
    """A small tensor in float32 on the part's device (kernels read sinks, gains and the like as float32 whatever
    the checkpoint stored)."""
    if t.dtype == torch.float32:
        return t.contiguous()
    if t.is_cuda and hasattr(env.ops, "cast"):
        out = torch.empty(t.shape, dtype=torch.float32, device=t.device)
        env.ops.cast(t.contiguous(), out)
        return out
    return t.to(torch.float32).contiguous()


class Norm(Part):
    def forward(self, residual, branch: Optional[Branch], ctx, rows=None) -> torch.Tensor:
        raise NotImplementedError

    @staticmethod
    def check_plain(branch: Optional[Branch], who: str, takes_bias: bool = False) -> None:
        """For norms that add one set of partials, unscaled: refuses a branch that asks for more."""
        if branch is not None and branch.bias is not None and not takes_bias:
            raise ValueError(f"{who}: the pending branch carries a bias; this norm adds outputs as they are")
        if branch is not None and (branch.more or branch.scale != 1.0 or branch.terms):
            raise ValueError(f"{who}: the pending branch carries several sublayers' outputs or a scale; "
                             f"this norm adds one output as it is")

    def forward_unscaled(self, residual, branch: Optional[Branch], ctx, rows=None):
        """``(x, row_scale)``: like ``forward``, but the norm may leave a per-row factor to the consumer
        (``row_scale``, a ``kernels.ops.RowScale``, or ``None`` when ``x`` is finished).  Called instead of
        ``forward`` for a consumer that sets ``TAKES_ROW_SCALE``."""
        return self.forward(residual, branch, ctx, rows), None


class Mixer(Part):
    TAKES_ROW_SCALE = False     # True: ``forward`` accepts ``row_scale=`` and applies it to the rows of ``x``

    def forward(self, x, ctx, cache) -> Branch:
        raise NotImplementedError

    def check_borrowed(self, need) -> None:
        """Called when the model is built for a mixer whose schedule entry reads another entry's cache
        (``cache_of``): ``need`` is what the owner keeps.  Raise ``ValueError`` if this mixer cannot read it."""


class FeedForward(Part):
    TAKES_ROW_SCALE = False     # as for ``Mixer``

    def forward(self, x, ctx) -> Branch:
        raise NotImplementedError


class PositionEncoding(Part):
    def prepare(self, max_positions: int) -> None:
        """Build tables for positions ``[0, max_positions)``.  May be called again with another number (a
        second engine on the same model): tables only grow, and one that a step may still read stays alive."""

    def limit(self) -> Optional[int]:
        """Positions the tables built so far cover (``None``: no limit)."""
        return None

    def rotation(self):
        """``None`` or a ``Rotation`` that a mixer applies to its queries and keys."""
        return None

    def query_scale(self):
        """``None`` or a float32 tensor with a number per position that a mixer multiplies its queries by."""
        return None

    def on_embeddings(self, residual, ctx) -> None:
        """Hook for encodings that are added to the embeddings (default: nothing)."""


class Block(Part):
    """``ROLES`` names the roles this arrangement has and the family each role's part is looked up in
    (``{"norm1": "norm", "mixer": "mixer", ...}``).  A layer's ``PartSpec`` may also carry its family
    itself; that wins, and lets a spec give a block a role that its class did not list."""

    ROLES: Dict[str, str] = {}

    def __init__(self, params, prefix, env, parts: Dict[str, Part]):
        super().__init__(params, prefix, env)
        self.parts = parts

    def forward(self, residual, pending: Optional[Branch], ctx, cache) -> Optional[Branch]:
        raise NotImplementedError

    def cache_parts(self):
        """The parts of this block that keep something per sequence (at most one: an entry of the run order
        has one cache unit)."""
        keepers = [p for p in self.parts.values() if p.cache_need() is not None]
        if len(keepers) > 1:
            raise ValueError("a block may hold only one part that keeps a cache or a state per sequence")
        return keepers

    def cache_need(self):
        keepers = self.cache_parts()
        return keepers[0].cache_need() if keepers else None


@dataclass
class BuildEnv:
    """What a part gets at construction: the compute dtype, the device, the kernels, shared encodings."""

    dtype: torch.dtype
    device: torch.device
    ops: Any
    encodings: Dict[str, PositionEncoding]


_REGISTRIES: Dict[str, Dict[str, Callable]] = {
    "norm": {}, "mixer": {}, "ffn": {}, "position": {}, "block": {}, "embedding": {}, "head": {}, "connection": {},
}


def register_part(family: str, kind: str, cls, *, replace: bool = False) -> None:
    """Make ``kind`` available to model specs; ``family`` is one of the registry names."""
    reg = _REGISTRIES[family]
    if kind in reg and not replace:
        raise ValueError(f"{family} part '{kind}' is already registered")
    reg[kind] = cls


def unregister_part(family: str, kind: str) -> None:
    _REGISTRIES[family].pop(kind, None)


def part_class(family: str, kind: str):
    reg = _REGISTRIES[family]
    if kind not in reg:
        raise KeyError(f"no {family} part named '{kind}' (known: {', '.join(sorted(reg)) or 'none'})")
    return reg[kind]


def part_families():
    return tuple(_REGISTRIES)
