"""Interfaces of the parts a model is put together from, and their registries.

A model is data: a :class:`ModelSpec` lists layers, each layer names its mixer, its
feed-forward, its norms and how they are arranged in a block, every one with its
sizes and constants as parameters; a schedule lists the order in which layers run.
Parts are looked up by name in the registries below, so a new mixer, feed-forward,
norm, position encoding or block arrangement is one class and one ``register``
call; no part knows which model it belongs to.

The reference builds its layers from fixed classes (src/model/layer.cuh:10-45,
src/model/attn.cuh:58-160, src/model/ffn.cuh:18-60); this file is the seam that
replaces that fixed structure.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Callable, Dict, Generic, List, Mapping, Optional, Sequence, Tuple, Type, TypeVar

import torch

T = TypeVar("T")

# Tokens per page of the key-value cache.  The one Python-side definition (cache and kernel wrappers import it); the
# kernels' own constant (csrc/common.cuh) is compared with it when the library is loaded.
PAGE_TOKENS = 64
# Query tokens per tile of the tiled prompt attention kernels (StepContext.q_tiles is made for this size).
QUERY_TILE_TOKENS = 64


class Registry(Generic[T]):
    """A table from a name to a class, with an error that lists what is known."""

    def __init__(self, what: str):
        self.what = what
        self._table: Dict[str, T] = {}

    def register(self, name: str) -> Callable[[T], T]:
        def deco(obj: T) -> T:
            if name in self._table and self._table[name] is not obj:
                raise KeyError(f"{self.what} '{name}' is already registered")
            self._table[name] = obj
            return obj
        return deco

    def unregister(self, name: str) -> None:
        self._table.pop(name, None)

    def get(self, name: str) -> T:
        try:
            return self._table[name]
        except KeyError:
            raise KeyError(f"unknown {self.what} '{name}'; known: {sorted(self._table)}") from None

    def names(self) -> List[str]:
        return sorted(self._table)

    def __contains__(self, name: str) -> bool:
        return name in self._table


# ---------------------------------------------------------------------------
# specifications (plain data)
# ---------------------------------------------------------------------------

@dataclass(frozen=True)
class PartSpec:
    """Which part (a registry name) and its sizes and constants."""

    kind: str
    params: Mapping[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class LayerSpec:
    """One layer: an arrangement (block) of a mixer, a feed-forward and their norms.

    ``prefix`` is the layer's part of the tensor names ("model.layers.3."); the
    names below it are given by ``names``: sub-part -> infix ("self_attn." ...).
    ``feed_forward`` and ``feed_forward_norm`` may be None: a layer of a mixer alone.
    """

    block: PartSpec
    mixer: PartSpec
    feed_forward: Optional[PartSpec]
    mixer_norm: PartSpec
    feed_forward_norm: Optional[PartSpec]
    prefix: str
    names: Mapping[str, str]


@dataclass(frozen=True)
class ScheduleEntry:
    """One run of a layer.  ``lane`` is the cache lane (keys, values, state) the run
    uses; ``writes_cache`` is False when the run only reads a lane an earlier run
    of this step has written (a layer that shares another layer's keys and values)."""

    layer: int
    lane: int
    writes_cache: bool = True
    # When not None, a pass through a repeated group of layers begins with this run, and the number is the pass's
    # (0, 1, ...): the model's ``pass_entry`` part then acts on the residual stream right before the run.
    enters_pass: Optional[int] = None


@dataclass(frozen=True)
class ModelSpec:
    architecture: str
    hidden_size: int
    vocab_size: int
    embedding: PartSpec
    layers: Sequence[LayerSpec]
    schedule: Sequence[ScheduleEntry]
    final_norm: PartSpec
    head: PartSpec
    embedding_name: str = "model.embed_tokens."
    final_norm_name: str = "model.norm."
    head_name: str = "lm_head."
    stop_token_ids: Sequence[int] = ()
    max_positions: int = 0
    # What happens to the residual stream where a run of the schedule ``enters_pass`` (None: nothing); its tensors
    # are named below ``pass_entry_name``.
    pass_entry: Optional[PartSpec] = None
    pass_entry_name: str = ""
    # Residual streams per token (0: the one plain stream).  With streams every token carries that many copies of the
    # residual vector, all equal to the embedding's output at the start; blocks that know of them read and write
    # ``ResidualStream.copies``, and the model's output norm sees their sum.
    streams: int = 0

    def n_lanes(self) -> int:
        return 1 + max(e.lane for e in self.schedule)


def default_schedule(n_layers: int) -> List[ScheduleEntry]:
    return [ScheduleEntry(layer=i, lane=i, writes_cache=True) for i in range(n_layers)]


@dataclass(frozen=True)
class WeightSpec:
    """Shape and role of one tensor.

    role "matrix": an operand of a matrix product or a lookup table of rows; held in
    the compute dtype.  role "vector": norm weights and other small tensors; a tensor
    stored in 32-bit stays in 32-bit.  role "table": integers, held as int32.
    """

    shape: Tuple[int, ...]
    role: str = "matrix"


@dataclass(frozen=True)
class CacheNeeds:
    """What one cache lane must hold for every sequence.

    kv_heads/head_dim: one key row and one value row per token and key-value head
    (0 heads = none).  window: None if every key stays needed, else the number of
    most recent tokens that do.  pooled_stride/pooled_kernel: an extra row per
    ``pooled_stride`` tokens (mean-pooled keys); 0 = none.  values: False when the
    lane keeps key rows only (a shared latent that keys and values are both made
    from).  value_dim: the size of a value row where it differs from a key row's (0: the same).  keep_first: with a
    window, the number of a sequence's first tokens that stay needed whatever the window.  state: tensors of fixed size per sequence, name -> (shape, dtype); they
    are zero when a sequence starts.
    """

    kv_heads: int = 0
    head_dim: int = 0
    window: Optional[int] = None
    pooled_stride: int = 0
    pooled_kernel: int = 0
    state: Mapping[str, Tuple[Tuple[int, ...], torch.dtype]] = field(default_factory=dict)
    values: bool = True
    value_dim: int = 0
    keep_first: int = 0

    def group_key(self) -> Tuple:
        return (self.kv_heads, self.head_dim, self.window, self.pooled_stride, self.pooled_kernel, self.values, self.value_dim,
                self.keep_first if self.window else 0)

    def seen_through(self, window: Optional[int]) -> "CacheNeeds":
        """The same needs when a further reader looks at the lane through ``window`` (None: at every key): the lane keeps
        what its widest reader sees."""
        if self.window is None or (window is not None and window <= self.window):
            return self
        return CacheNeeds(self.kv_heads, self.head_dim, window, self.pooled_stride, self.pooled_kernel, self.state, self.values,
                          self.value_dim, self.keep_first)

    def with_state(self, more: Mapping[str, Tuple[Tuple[int, ...], torch.dtype]]) -> "CacheNeeds":
        """The same needs with further per-sequence tensors (a block adds its own to its mixer's)."""
        both = dict(self.state)
        for name, what in more.items():
            if name in both:
                raise ValueError(f"per-sequence state '{name}' is declared twice for one lane")
            both[name] = what
        return CacheNeeds(self.kv_heads, self.head_dim, self.window, self.pooled_stride, self.pooled_kernel, both, self.values,
                          self.value_dim, self.keep_first)


# ---------------------------------------------------------------------------
# part interfaces
# ---------------------------------------------------------------------------

class Part:
    """Common to all parts: declared weights, and loading them.

    ``ops`` is the kernel library bound to a compute dtype (see cpmcu_b200.ops); a
    part calls kernels only through it.
    """

    def __init__(self, ops):
        self.ops = ops

    def weight_specs(self) -> Dict[str, WeightSpec]:
        """Tensor names below this part's prefix -> shape and role."""
        return {}

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Receives exactly the tensors of ``weight_specs`` (already on the device)."""

    def weight_bytes(self) -> int:
        """Bytes of weights one step reads (each tensor once)."""
        return 0

    # True if ``forward`` reads nothing of the batch on the host but ``n_tokens``, ``n_seqs``, ``q_lens`` and the
    # upper bound ``max_kv_len``, for prompts too: such a part can be recorded into a graph for a prompt chunk
    # (a part that walks ``ctx.slots`` or ``ctx.kv_lens`` on the host cannot; the default is the safe answer).
    recordable_prompt = False


class Norm(Part):
    def forward(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """x: fp32 [tokens, hidden] residual stream -> normed [tokens or len(rows), hidden] in compute dtype."""
        raise NotImplementedError

    def add_forward(self, x: torch.Tensor, delta: torch.Tensor, scale: float,
                    rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """x += scale*delta (written back unless ``rows`` is given), then forward."""
        raise NotImplementedError


class PositionEncoding(Part):
    """Position information for a mixer.

    A rotary encoding that the fused rotate-and-store kernel can apply returns its
    table from ``rotary()``; any other encoding returns None there and transforms
    the queries and keys itself in ``apply``.
    """

    def rotary(self) -> Optional[Tuple[torch.Tensor, float, int]]:
        """(inv_freq fp32 [rot_dim/2], magnitude factor for cos and sin, rot_dim) or None."""
        return None

    def apply(self, ctx: "StepContext", q: torch.Tensor, k: torch.Tensor) -> None:
        """In place on q [tokens, heads, d] and k [tokens, kv_heads, d] (views with strides)."""


class Mixer(Part):
    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds()

    def forward(self, ctx: "StepContext", y: torch.Tensor, lane, writes_cache: bool) -> torch.Tensor:
        """y: normed [tokens, hidden] (compute dtype) -> [tokens, hidden]."""
        raise NotImplementedError

    def cache_bytes_read(self, kv_len: int) -> int:
        """Bytes of cache one decode step of a sequence with ``kv_len`` keys has to read."""
        return 0


class FeedForward(Part):
    def forward(self, ctx: "StepContext", y: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError


class ResidualStream:
    """The fp32 residual sum of a step, with the last part's output still to be added.

    The addition of a part's output is deferred so that the next norm does it in the
    same kernel (the reference fuses the add into its norm kernel too:
    src/model/norm.cuh:53-99); the sum itself is always kept and formed in 32-bit.
    """

    def __init__(self, ops, x: torch.Tensor, narrow: Optional[torch.Tensor] = None):
        self.ops = ops
        self.x = x
        # x in the compute dtype, where the kernel that wrote x last left that too (None: nobody did)
        self.narrow: Optional[torch.Tensor] = narrow
        self.pending: Optional[torch.Tensor] = None
        self.pending2: Optional[torch.Tensor] = None       # a second output with the same factor (two sublayers side by side)
        self.pending_scale: float = 1.0
        # several streams per token: fp32 [tokens, streams, hidden], and the last sublayer's write still to be done
        # (its output, the mix matrix, the output weights), which the next read performs in the same pass
        self.copies: Optional[torch.Tensor] = None
        self.pending_write = None

    def fan_out(self, n_streams: int) -> None:
        """From here on the token carries ``n_streams`` residual vectors, each a copy of x."""
        self.flush()
        self.copies = self.ops.hyper_fan_out(self.x, int(n_streams))

    def add(self, delta: torch.Tensor, scale: float = 1.0, second: Optional[torch.Tensor] = None) -> None:
        """x += scale * delta (+ scale * second), deferred to the next norm's pass or the next ``flush``."""
        self.flush()
        self.narrow = None
        self.pending = delta
        self.pending2 = second
        self.pending_scale = float(scale)

    def flush(self) -> torch.Tensor:
        if self.copies is not None:
            # x becomes the sum of the streams (after the write that is still due)
            self.ops.hyper_step(self.copies, write=self.pending_write, total=self.x)
            self.pending_write = None
            return self.x
        if self.pending is not None:
            self.ops.residual_add(self.x, self.pending, self.pending_scale)
            if self.pending2 is not None:
                self.ops.residual_add(self.x, self.pending2, self.pending_scale)
            self.pending = self.pending2 = None
        return self.x

    def itself(self) -> torch.Tensor:
        """The stream in the compute dtype, for a sublayer that reads it without a norm in front."""
        x = self.flush()
        if self.narrow is None or self.copies is not None:
            self.narrow = self.ops.narrowed(x)
        return self.narrow

    def normed(self, norm: Norm, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        if self.copies is not None:
            return norm.forward(self.flush(), rows)
        if self.pending is None:
            return norm.forward(self.x, rows)
        if self.pending2 is not None:
            if not getattr(norm, "takes_two_addends", False):
                return norm.forward(self.flush(), rows)
            y = norm.add_forward(self.x, self.pending, self.pending_scale, rows, second=self.pending2)
        else:
            y = norm.add_forward(self.x, self.pending, self.pending_scale, rows)
        if rows is None:
            self.pending = self.pending2 = None
        return y


class Block(Part):
    """An arrangement of a mixer, a feed-forward and norms around the residual stream."""

    def __init__(self, ops, mixer: Mixer, feed_forward: Optional[FeedForward], mixer_norm: Norm,
                 feed_forward_norm: Optional[Norm], names: Mapping[str, str]):
        super().__init__(ops)
        self.mixer = mixer
        self.feed_forward = feed_forward
        self.mixer_norm = mixer_norm
        self.feed_forward_norm = feed_forward_norm
        self.names = dict(names)

    def sub_parts(self) -> List[Tuple[str, Part]]:
        parts = [
            (self.names.get("mixer_norm", "mixer_norm."), self.mixer_norm),
            (self.names.get("mixer", "mixer."), self.mixer),
            (self.names.get("feed_forward_norm", "feed_forward_norm."), self.feed_forward_norm),
            (self.names.get("feed_forward", "feed_forward."), self.feed_forward),
        ]
        return [(infix, part) for infix, part in parts if part is not None]      # a layer may have no feed-forward

    def weight_specs(self) -> Dict[str, WeightSpec]:
        out: Dict[str, WeightSpec] = {}
        for infix, part in self.sub_parts():
            for name, spec in part.weight_specs().items():
                out[infix + name] = spec
        return out

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        for infix, part in self.sub_parts():
            names = part.weight_specs()
            part.load_weights({n: tensors[infix + n] for n in names})

    def weight_bytes(self) -> int:
        return sum(p.weight_bytes() for _, p in self.sub_parts())

    def cache_needs(self) -> CacheNeeds:
        """What a run of this layer keeps per sequence: its mixer's needs, plus whatever the arrangement itself
        carries from token to token."""
        return self.mixer.cache_needs()

    def forward(self, ctx: "StepContext", stream: ResidualStream, lane, writes_cache: bool) -> None:
        raise NotImplementedError


MIXERS: Registry[Type[Mixer]] = Registry("mixer")
FEED_FORWARDS: Registry[Type[FeedForward]] = Registry("feed-forward")
NORMS: Registry[Type[Norm]] = Registry("norm")
POSITIONS: Registry[Type[PositionEncoding]] = Registry("position encoding")
BLOCKS: Registry[Type[Block]] = Registry("block")


class PassEntry(Part):
    """Acts on the residual stream where a pass through a repeated group of layers begins."""

    def forward(self, ctx: "StepContext", stream: ResidualStream, number: int, embedded: torch.Tensor) -> None:
        """``number``: the pass's (0, 1, ...); ``embedded``: the stream as the embedding left it (fp32, read only)."""
        raise NotImplementedError


PASS_ENTRIES: Registry[Type[PassEntry]] = Registry("pass entry")


def build_part(registry: Registry, spec: PartSpec, ops):
    cls = registry.get(spec.kind)
    try:
        return cls(ops, **dict(spec.params))
    except TypeError as e:
        raise TypeError(f"{registry.what} '{spec.kind}': bad parameters {sorted(spec.params)} ({e})") from None


def build_block(spec: LayerSpec, ops) -> Block:
    cls = BLOCKS.get(spec.block.kind)
    return cls(
        ops,
        mixer=build_part(MIXERS, spec.mixer, ops),
        feed_forward=build_part(FEED_FORWARDS, spec.feed_forward, ops) if spec.feed_forward is not None else None,
        mixer_norm=build_part(NORMS, spec.mixer_norm, ops),
        feed_forward_norm=build_part(NORMS, spec.feed_forward_norm, ops) if spec.feed_forward_norm is not None else None,
        names=spec.names,
        **dict(spec.block.params),
    )


# ---------------------------------------------------------------------------
# what a step hands to the parts
# ---------------------------------------------------------------------------

@dataclass
class StepContext:
    """One step's batch, as the parts see it.

    Host-side lists describe the batch for Python-level decisions; the device
    tensors are what kernels read.  Both are filled whenever a step runs eagerly:
    by the step function, and by the decode runner without a graph (its padding
    entries appear as sequences of one key in a scratch slot).

    In a captured step (``captured`` True: a decode step, or a prompt chunk of one
    sequence when every part of the model is ``recordable_prompt``) the device tensors are fixed
    buffers whose contents change between replays; the recording is made once, on
    padding entries only, and replayed for any batch.  A part may then read only:
    ``n_tokens``, ``n_seqs`` (the bucket size), ``is_decode``, ``q_lens`` (all 1, or the chunk's size),
    ``max_q_len``, ``max_kv_len`` (the cache's capacity per sequence, an upper
    bound), the device tensors, ``cache`` and its lanes.  ``kv_lens`` and ``slots`` are
    empty; everything that depends on a sequence (its slot, its length, its state
    in ``lane.state[name][slot]``) has to be reached on the device through
    ``slot_dev`` and ``kv_len_dev``, with operations that can be recorded (no
    host read, no data-dependent shapes).
    """

    n_tokens: int
    n_seqs: int
    is_decode: bool                      # every sequence brings exactly one token
    captured: bool
    # host
    q_lens: List[int]
    kv_lens: List[int]                   # keys per sequence after this step's tokens are stored
    slots: List[int]
    max_q_len: int
    max_kv_len: int
    # device (int32)
    token_ids: torch.Tensor              # [tokens]
    positions: torch.Tensor              # [tokens]
    token_seq: torch.Tensor              # [tokens] index of the token's sequence in this batch
    cu_q: torch.Tensor                   # [seqs+1] offsets of the sequences in the token axis
    kv_len_dev: torch.Tensor             # [seqs]
    slot_dev: torch.Tensor               # [seqs]
    cache: Any = None                    # cpmcu_b200.cache.Cache
    workspace: Any = None                # per-engine scratch tensors by name
    # Query tiles for mixers that work on tiles of QUERY_TILE_TOKENS consecutive tokens of one sequence (the tiled
    # prompt attention): (tile -> sequence index int32 [tiles], tile -> first token inside the sequence's tokens of
    # this step int32 [tiles], number of tiles); None when the step's maker gives none (a mixer then falls back to
    # a kernel that needs no tiles).
    q_tiles: Optional[Tuple[torch.Tensor, torch.Tensor, int]] = None
    extras: Dict[str, Any] = field(default_factory=dict)
