"""What a layer is made of, in general terms.

A model is a list of *blocks*; a block arranges a *mixer* (attention here), a *feed-forward*
and *norms*; a mixer may use a *position encoding*.  Every part takes its sizes and constants
as constructor arguments and is chosen by the architecture's builder layer by layer, by name,
from the registries below.  No part knows which model it is in: it sees its own parameters and
the ``StepContext`` of the step being run.

Interfaces
----------
``Part``            parameters declared as ``ParamSpec``s (name, shape, init), filled by the loader.
``Mixer``           ``forward(h, ctx, site) -> y``; declares ``cache_spec()`` (paged keys/values)
                    and/or ``state_spec()`` (fixed-size per-request state).
``FeedForward``     ``forward(h, ctx) -> y``.
``Norm``            ``forward(x, pending, out, rows=None)``: adds the pending sub-layer output
                    into the float32 residual stream ``x`` and writes the normalised rows.
``PositionEncoding`` used by a mixer; the rotary one exposes ``inv_freq``/``rotary_dim``/pairing.
``Block``           ``forward(x, pending, ctx, site) -> pending'`` (residual handling is the
                    block's business: pre-norm here).
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass, field
from typing import Any, Callable, Dict, List, Optional, Sequence, Tuple

import torch


# ------------------------------------------------------------------------------ parameters

@dataclass
class ParamSpec:
    """One tensor a part owns.  ``init``: ("normal", std) | ("ones",) | ("ones_jitter", std) | ("eye_jitter", std)."""
    name: str
    shape: Tuple[int, ...]
    init: Tuple = ("normal", 0.02)
    kind: str = "matrix"            # "matrix" | "vector" | "table"


class Part:
    """Base of every part: named parameters, named children.

    ``capturable``: a step that contains the part may be recorded into a CUDA graph and replayed.
    That asks three things of ``forward``: it only enqueues device work (no host synchronisation,
    no host-side reading of device data); everything that changes from step to step reaches it
    through device memory at fixed addresses (the ``StepContext``'s index tensors, the cache, state
    slabs), never through Python values or freshly computed shapes; and a replay does exactly what
    the recorded call did, once -- a part with state of its own may update it in place, the engine
    runs every step exactly once, the step that is recorded included.  A part that cannot promise
    this sets it to False and the engine replays no graphs."""

    capturable = True

    def __init__(self) -> None:
        self._specs: Dict[str, ParamSpec] = {}
        self._params: Dict[str, Optional[torch.Tensor]] = {}
        self._children: Dict[str, "Part"] = {}

    # declaration
    def declare(self, name: str, shape: Sequence[int], init: Tuple = ("normal", 0.02),
                kind: str = "matrix") -> None:
        self._specs[name] = ParamSpec(name, tuple(int(s) for s in shape), init, kind)
        self._params[name] = None

    def add_child(self, name: str, part: "Part") -> "Part":
        self._children[name] = part
        return part

    # access
    def param_specs(self) -> Dict[str, ParamSpec]:
        return dict(self._specs)

    def children(self) -> Dict[str, "Part"]:
        return dict(self._children)

    def set_param(self, name: str, tensor: torch.Tensor) -> None:
        spec = self._specs[name]
        if tuple(tensor.shape) != spec.shape:
            raise ValueError(f"{type(self).__name__}.{name}: shape {tuple(tensor.shape)} != {spec.shape}")
        self._params[name] = tensor
        self.on_param_set(name, tensor)

    def on_param_set(self, name: str, tensor: torch.Tensor) -> None:   # hook for subclasses
        pass

    def param(self, name: str) -> torch.Tensor:
        t = self._params[name]
        if t is None:
            raise RuntimeError(f"{type(self).__name__}.{name} has not been loaded")
        return t

    def named_parts(self, prefix: str = ""):
        yield prefix, self
        for n, c in self._children.items():
            yield from c.named_parts(f"{prefix}.{n}" if prefix else n)

    def prepare(self, device: torch.device, dtype: torch.dtype) -> None:
        """Called once after loading: build device-side constants (tables and the like)."""
        for c in self._children.values():
            c.prepare(device, dtype)


# ----------------------------------------------------------------------------- cache needs

@dataclass(frozen=True)
class CacheSpec:
    """Paged keys and values a mixer needs per layer: geometry and how long keys live."""
    num_kv_heads: int
    head_dim: int
    window: int = 0                 # 0: every key is kept; w: only the last w positions
    values: bool = True             # False: one pool only (a mixer that derives keys AND values from what it caches)
    chunk: int = 0                  # c: position i needs only the keys of its own chunk, j >= i - i % c


@dataclass(frozen=True)
class StateSpec:
    """Fixed-size per-request state a mixer keeps per layer: one tensor [slots, *shape]."""
    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class LayerCall:
    """One entry of the model's run order: which layer runs, and whose cache it uses.

    ``cache_of``: None = this call site has a cache of its own (and writes it); an integer =
    the index (in the run order) of an earlier call site whose cache it reads without writing.
    ``enter``: a part that works on the residual stream before the layer runs (``StreamPart``) with
    the argument it is called with, e.g. the entry of a span of layers that runs several times and the
    number of the pass."""
    layer: int
    cache_of: Optional[int] = None
    enter: Optional[Tuple[Any, Any]] = None


# -------------------------------------------------------------------------------- contexts

@dataclass
class GroupView:
    """What a step sees of one layer group: the step's page tables and slot mapping."""
    block_tables: torch.Tensor      # int32 [S, max_blocks]
    slot_mapping: torch.Tensor      # int32 [T]
    block_size: int
    window: int


@dataclass
class SiteCache:
    """The cache of one call site: paged K/V of its layer (a view into the group pool) and/or
    its state slab."""
    group: int = -1
    k: Optional[torch.Tensor] = None        # [pages, nkv, block, hd]
    v: Optional[torch.Tensor] = None        # None when the group's spec keeps no values
    writes: bool = True
    state: Optional[torch.Tensor] = None    # [slots, *shape], the mixer's
    block_state: Optional[torch.Tensor] = None   # [slots, *shape], the block's own (see Block.state_spec)
    shares: Optional[tuple] = None          # the site as the parts of a composed mixer see it (made by that mixer, once)


@dataclass
class StepContext:
    """Everything a part may read about the step being run.  All index tensors are int32 on
    the device; the host-side counts are plain ints."""
    rows: int                        # T (with padding)
    seqs: int                        # S (with padding)
    decode_seqs: int                 # entries [0, decode_seqs) are single rows; rows [0, decode_seqs)
    prefill_rows: int
    prefill_tiles: int
    tile_rows: int
    max_ctx: int
    max_decode_ctx: int
    max_q_len: int
    tokens: torch.Tensor
    positions: torch.Tensor
    row_seq: torch.Tensor
    seq_q_start: torch.Tensor
    seq_q_len: torch.Tensor
    seq_ctx_len: torch.Tensor
    seq_state_slot: torch.Tensor
    tile_seq: torch.Tensor
    tile_q0: torch.Tensor
    logit_rows: torch.Tensor
    groups: List[GroupView]
    dtype: torch.dtype               # storage dtype of activations
    workspace: Any = None            # per-engine scratch provider (see engine.runner.Workspace)
    options: Dict[str, Any] = field(default_factory=dict)
    prev_tokens: Optional[torch.Tensor] = None   # per row: the request's token one position earlier (-1 at position 0)
    h_stream: Optional[torch.Tensor] = None      # storage-dtype copy of the residual stream, kept current by blocks
                                                 # whose sublayers read the stream itself (None: nobody keeps one)
    shared: Dict[str, Any] = field(default_factory=dict)   # what a layer leaves for later layers of the SAME step
                                                           # (per-row tensors, e.g. an early layer's values)


# ------------------------------------------------------------------------------ registries

class Registry:
    def __init__(self, what: str) -> None:
        self.what = what
        self._items: Dict[str, Callable[..., Any]] = {}

    def register(self, name: str, factory: Callable[..., Any] = None, *, replace: bool = False):
        def deco(f):
            if name in self._items and not replace:
                raise ValueError(f"{self.what} '{name}' is already registered")
            self._items[name] = f
            return f
        return deco(factory) if factory is not None else deco

    def get(self, name: str) -> Callable[..., Any]:
        if name not in self._items:
            raise KeyError(f"unknown {self.what} '{name}'; registered: {', '.join(sorted(self._items))}")
        return self._items[name]

    def build(self, name: str, **kwargs):
        return self.get(name)(**kwargs)

    def names(self) -> List[str]:
        return sorted(self._items)


MIXERS = Registry("mixer")
FEED_FORWARDS = Registry("feed-forward")
NORMS = Registry("norm")
POSITION_ENCODINGS = Registry("position encoding")
BLOCKS = Registry("block")


class Mixer(Part):
    """``forward(h, ctx, site)`` does the whole of it.  A mixer whose work falls into the stages below sets ``staged``: two
    such mixers that read the same rows can share the launches of the first, second and fourth (``side_by_side``), and
    ``forward_staged`` is the mixer alone.

        projection        the ``Linear`` whose float32 rows hold all it needs of h
        begin(proj, base, dtype, ctx, site) -> work     ``work.segments`` (``kernels.library.HeadSegment``s, columns from ``base``
                          on), ``work.conv`` (a ``HeadConv`` or None): what one ``prepare_heads`` launch has to do
        mix(work)         -> ``kernels.library.GateSegment``: attention or recurrence; what a ``gate_heads`` launch has to do
        finish(work)      -> the output product of the gated heads, float32"""
    staged = False

    def forward_staged(self, h: torch.Tensor, ctx: StepContext, site: SiteCache) -> torch.Tensor:
        from ..kernels import library as K
        proj = self.projection.forward(h, ctx, out_dtype=torch.float32)
        work = self.begin(proj, 0, h.dtype, ctx, site)
        run_prepare(proj, [work], h.dtype, ctx)
        K.gate_heads(proj, [self.mix(work)])
        return self.finish(work)

    def cache_spec(self) -> Optional[CacheSpec]:
        return None

    def state_spec(self) -> Optional[StateSpec]:
        return None

    def forward(self, h: torch.Tensor, ctx: StepContext, site: SiteCache) -> torch.Tensor:
        raise NotImplementedError


class StagedWork:
    """What a staged mixer keeps of one call (see ``Mixer``); ``block_size`` and ``slot_mapping`` are those of its page group."""

    def __init__(self, proj: torch.Tensor, base: int, dtype: torch.dtype, ctx: StepContext, site: SiteCache) -> None:
        self.proj, self.base, self.dtype, self.ctx, self.site = proj, base, dtype, ctx, site
        self.segments: List[Any] = []
        self.conv: Any = None
        self.slot_mapping: Optional[torch.Tensor] = None
        self.block_size = 1
        self.out: Optional[torch.Tensor] = None          # the gated heads


def run_prepare(proj: torch.Tensor, works, dtype: torch.dtype, ctx: StepContext) -> None:
    """One ``prepare_heads`` launch for the given mixers (at most one of them convolves, at most one writes pages)."""
    from ..kernels import library as K
    segments = [s for w in works for s in w.segments]
    if not segments:
        return
    conv = next((w.conv for w in works if w.conv is not None), None)
    paged = next((w for w in works if w.slot_mapping is not None), None)
    K.prepare_heads(proj, segments, ctx, dtype, conv, paged.slot_mapping if paged else None,
                    paged.block_size if paged else 1)


class FeedForward(Part):
    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        raise NotImplementedError


class Norm(Part):
    def forward(self, x: torch.Tensor, pending: Optional[torch.Tensor], out: torch.Tensor,
                rows: Optional[torch.Tensor] = None) -> None:
        raise NotImplementedError


class PositionEncoding(Part):
    pass


class ClosingNorm:
    """A sublayer's float32 output ``y`` (or a ``NormedSum`` / ``ExpertSum`` that is still to be formed) that is to be added
    to the stream through an RMS norm: x += multiplier * y / sqrt(mean(y^2) + eps).  A block may hand this on as its pending value so that the
    reader of the stream applies it in the same kernel as its own opening norm."""
    __slots__ = ("y", "multiplier", "eps")

    def __init__(self, y: torch.Tensor, multiplier: torch.Tensor, eps: float) -> None:
        self.y, self.multiplier, self.eps = y, multiplier, float(eps)


class NormedSum:
    """A mixer's output made of two branches before its sum: sum of multiplier * y / sqrt(mean(y^2) + eps) over
    ``branches``, two (float32 [rows, width], float32 multiplier [width]) pairs.  The kernel that applies the norm behind
    the mixer forms the sum in the same pass; ``formed`` forms it by itself."""
    __slots__ = ("branches", "eps")

    def __init__(self, branches, eps: float) -> None:
        self.branches, self.eps = tuple(branches), float(eps)

    def formed(self) -> torch.Tensor:
        from ..kernels import library as K
        out = torch.zeros_like(self.branches[0][0])
        for y, multiplier in self.branches:
            K.norm_post_pre(out, y, multiplier, None, None, self.eps)
        return out


class ExpertSum:
    """A routed feed-forward's output before its weighted sum: ``y`` float32 [rows * top, width] in the order of the
    sorted pairs, ``wt`` float32 [rows, top], ``work`` the sort's scratch (it holds every pair's place).  A block may hand
    this on as pending, so that the reader of the stream forms the sum in its own kernel."""
    __slots__ = ("y", "work", "wt", "experts")

    def __init__(self, y: torch.Tensor, work: torch.Tensor, wt: torch.Tensor, experts: int) -> None:
        self.y, self.work, self.wt, self.experts = y, work, wt, int(experts)

    def place(self) -> ctypes.c_void_p:
        """Where every (row, choice) pair's row of ``y`` is listed, as the experts' sort leaves it."""
        return ctypes.c_void_p(self.work.data_ptr() + 4 * (self.experts + 2 + self.wt.numel()))

    def combined(self) -> torch.Tensor:
        from ..kernels import library as K
        out = torch.empty((self.wt.shape[0], self.y.shape[1]), dtype=torch.float32, device=self.y.device)
        K.moe_combine(self.y, self.work, self.wt, self.experts, None, None, out)
        return out


def split_pending(pending):
    """What a layer left pending as ([(float32 tensor, scale), ...], one ``ExpertSum`` or None)."""
    if pending is None:
        return [], None
    items = list(pending) if isinstance(pending, (list, tuple)) else [pending if isinstance(pending, ExpertSum) else (pending, 1.0)]
    dense, experts = [], None
    for item in items:
        if not isinstance(item, ExpertSum):
            t, scale = item
            dense.append((t if t.dtype == torch.float32 else t.float(), scale))
        elif experts is None:
            experts = item
        else:
            dense.append((item.combined(), 1.0))
    return dense, experts


def settle(x: torch.Tensor, pending) -> None:
    """Brings the float32 stream ``x`` up to date with what the layer before left pending: nothing, a tensor
    to add, a ``ClosingNorm``, an ``ExpertSum``, or a list of (tensor, scale) pairs and ``ExpertSum``s."""
    from ..kernels import library as K
    if pending is None:
        return
    if isinstance(pending, (list, tuple)):
        for item in pending:
            if isinstance(item, ExpertSum):
                settle(x, item)
            else:
                settle(x, item[0] if item[1] == 1.0 else item[0] * item[1])
        return
    if isinstance(pending, ExpertSum):
        K.add_residual(x, pending.combined())
        return
    if isinstance(pending, ClosingNorm):
        K.norm_post_pre(x, pending.y, pending.multiplier, None, None, pending.eps)
    else:
        K.add_residual(x, pending)


class StreamPart(Part):
    """A part between two layers: ``forward(x, pending, ctx, arg) -> (x', pending')`` takes the float32
    residual stream (and what the layer before left pending) and returns the stream the next layer reads."""

    def forward(self, x: torch.Tensor, pending, ctx: StepContext, arg=None):
        raise NotImplementedError


class Block(Part):
    """``moves_stream``: ``forward`` leaves x as it is and returns (x', pending') with the stream in a new tensor
    (a kernel that reads neighbouring rows of the old stream cannot write the new one in place).
    ``state_spec``: fixed-size per-request state that the arrangement itself keeps, beside the mixer's; it arrives
    as ``site.block_state``."""
    mixer: Mixer
    moves_stream = False

    def state_spec(self) -> Optional[StateSpec]:
        return None

    def forward(self, x: torch.Tensor, pending: Optional[torch.Tensor], ctx: StepContext,
                site: SiteCache) -> torch.Tensor:
        raise NotImplementedError
