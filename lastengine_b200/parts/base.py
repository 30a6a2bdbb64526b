"""What a part of a layer is, and what a model is made of.

A layer is put together from parts: a mixer (attention, short convolution, ...), a
feed-forward (dense or experts), norms and a position encoding, arranged by a block.
Each part gets its sizes and constants as constructor arguments and knows nothing of the
model around it.  Which parts a layer has is data (`PartSpec`), chosen layer by layer; the
order in which layers run is data too (`ScheduleEntry`).

Interfaces
----------
Every part:
    tensors()  -> {relative name: TensorSpec}     what it reads from the checkpoint
    load(tensors, env)                             takes its tensors (already on the device,
                                                   in the dtype of their role) and may fuse them
Mixer:
    cache_spec() -> KVSpec | LatentSpec | StateSpec what it keeps per sequence (or a tuple of at most one
                    | (KVSpec, StateSpec, ...) | None KVSpec and any states of different shapes)
    forward(h, out, accumulate, batch, cache, env) h: [rows, hidden] normed input in the
                                                   activation dtype; writes (or adds) its
                                                   result into the float tensor `out`
FeedForward:
    forward(h, out, accumulate, batch, env)
Norm:
    forward(out, x, rows=None, add=False)          x float; out in any activation dtype
Embedding:
    forward(x, tokens, batch=...)                  x: float [rows, hidden], written.  One that keeps state per sequence has
                                                   a cache_spec() and gets its view as `cache=`
PositionEncoding:
    fused_rotary() -> (inv_freq, rope_dim, neox)   a rotation that the mixer's kernel applies itself
                      | None                       while it norms q and k and stores k and v, or
    apply(q, k, row_pos)                           any other encoding, in place on the normed
                                                   q [rows, heads, head_dim] and k [rows, kv heads, head_dim]
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

import torch

# roles decide the random initialisation and the dtype a tensor is kept in
MATRIX = "matrix"        # operand of a matrix product: kept in the compute dtype
EMBEDDING = "embedding"  # token table: compute dtype
NORM = "norm"            # norm weight: kept float
NORM_AROUND_ZERO = "norm0"   # norm weight stored around zero (the factor is 1 + w): kept float
VECTOR = "vector"        # small per-channel parameters (conv taps, router rows): kept float
BIAS = "bias"            # additive terms: kept float

FLOAT_ROLES = (NORM, NORM_AROUND_ZERO, VECTOR, BIAS)


@dataclass(frozen=True)
class TensorSpec:
    shape: tuple[int, ...]
    role: str
    std: float | None = None      # random init: normal(0, std); None: the model's default
    optional: bool = False        # may be absent from the checkpoint
    shared_name: str | None = None  # the tensor's full name where it belongs to the model, not to the
                                    # part's prefix (several parts may then name the same tensor)
    free: int | None = None       # a size the checkpoint decides stands as -1 in `shape`; random weights take this one

    def fits(self, found: tuple[int, ...]) -> bool:
        """Whether a stored tensor of shape `found` is one of this spec (-1 takes any size)."""
        return len(found) == len(self.shape) and all(s in (-1, int(f)) for s, f in zip(self.shape, found))

    def concrete_shape(self) -> tuple[int, ...]:
        """The shape random weights are made with."""
        if -1 in self.shape and self.free is None:
            raise ValueError(f"a tensor of shape {self.shape} has a size only a checkpoint gives")
        return tuple(self.free if s == -1 else s for s in self.shape)


@dataclass(frozen=True)
class KVSpec:
    """Keys and values that grow with the sequence; `window` > 0 keeps only the last ones, `chunk` > 0 only those
    of the chunk of that many positions (counted from the sequence's first) the next position lies in.
    `v_head_dim`: width of a value head where it differs from a key head's (None: the same).
    `pool` > 0: beside them one pooled key and value row for every complete block of `pool` positions,
    in pages of their own (block b in row b); they stay when the window has let the block's positions go."""
    n_kv_heads: int
    head_dim: int
    window: int = 0
    v_head_dim: int | None = None
    pool: int = 0
    chunk: int = 0

    @property
    def value_dim(self) -> int:
        return self.head_dim if self.v_head_dim is None else self.v_head_dim


@dataclass(frozen=True)
class LatentSpec:
    """One row per position that stands for every head's key and value: a latent vector of `rank`
    numbers followed by `rope_dim` numbers of a rotated key part shared by all heads.  Paged like keys
    and values (one pool of rows `[position][rank + rope_dim]`, nothing stored apart for the values); `window`
    and `chunk` as there."""
    rank: int
    rope_dim: int
    window: int = 0
    chunk: int = 0

    # how the cache's page groups see it: one "head" whose key row is the whole cached row
    n_kv_heads = 1
    value_dim = 0

    @property
    def head_dim(self) -> int:
        return self.rank + self.rope_dim


@dataclass(frozen=True)
class StateSpec:
    """State of fixed size per sequence, zero when the sequence starts."""
    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class PartSpec:
    kind: str                      # name in the registry of its family
    params: dict[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class LayerSpec:
    prefix: str                    # tensor-name prefix of the layer, e.g. "layers.3"
    mixer: PartSpec
    ffn: PartSpec | None           # None: the layer has no feed-forward sublayer (a block arrangement that allows it)
    mixer_norm: PartSpec
    ffn_norm: PartSpec | None
    post_mixer_norm: PartSpec | None = None
    post_ffn_norm: PartSpec | None = None
    block: str = "pre_norm_residual"
    # tensor-name prefixes of the parts, relative to `prefix`
    names: dict[str, str] = field(default_factory=dict)
    # gates on the sublayers' results, by the name under which the block arrangement takes them
    gates: dict[str, PartSpec] = field(default_factory=dict)
    # constants of the block arrangement itself (keyword arguments of its class)
    block_params: dict[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class StreamAdd:
    """What happens to the residual stream right before a schedule entry runs: the embedding output (the stream
    as it was before the first entry) and/or one row of a model-wide table is added; with `matrix` the stream first
    becomes W [stream ; embedding output], and the row is added to that."""
    before: int                    # index into the schedule
    embedding: bool = False
    table: str | None = None       # canonical tensor name of a [rows, hidden] table
    row: int = 0
    matrix: str | None = None      # canonical tensor name of a [hidden, 2 hidden] matrix


@dataclass(frozen=True)
class ScheduleEntry:
    """One step of the layer order: run `layer` with the cache entry `cache`.

    By default entry i runs layer i with its own cache entry i.  Naming a layer twice runs
    its weights twice; `cache` pointing at an earlier entry with `writes_cache=False` lets a
    layer read what that entry stored instead of storing its own.
    """
    layer: int
    cache: int | None = None
    writes_cache: bool = True


@dataclass
class ModelPlan:
    """Everything needed to build a model: parts, their order, and the tensor names."""
    architecture: str
    hidden_size: int
    vocab_size: int
    embedding: PartSpec
    final_norm: PartSpec
    head: PartSpec
    layers: list[LayerSpec]
    schedule: list[ScheduleEntry]
    init_std: float = 0.02
    init_stds: dict[str, float] = field(default_factory=dict)   # tensor-name suffix -> std, before init_std
    eos_token_ids: tuple[int, ...] = ()
    names: dict[str, str] = field(default_factory=dict)   # prefixes of embedding / final_norm / head
    tensor_aliases: Any = None     # callable: checkpoint name -> canonical name (or None)
    unused_tensors: tuple[str, ...] = ()   # canonical names a checkpoint of the architecture may hold that this
                                           # model has no use for (an optional tensor of a part no layer has): skipped
    stream_adds: tuple[StreamAdd, ...] = ()     # additions to the residual stream between schedule entries
    stream_tables: dict[str, tuple[int, ...]] = field(default_factory=dict)   # canonical name -> shape of their tables
    stream_matrices: dict[str, tuple[int, ...]] = field(default_factory=dict)   # canonical name -> shape of their matrices
    max_positions: int | None = None   # the longest sequence the model takes (a table of learned positions); None: no limit
    checkpoint_names: Any = None   # callable: canonical name -> name in a checkpoint (the inverse of
                                   # tensor_aliases; None: "model." in front of everything but the head)

    def __post_init__(self):
        n = len(self.layers)
        for i, e in enumerate(self.schedule):
            if not 0 <= e.layer < n:
                raise ValueError(f"schedule[{i}] names layer {e.layer}, the model has {n}")
            c = i if e.cache is None else e.cache
            if not 0 <= c < len(self.schedule):
                raise ValueError(f"schedule[{i}] names cache entry {c}, outside the schedule")
            if not e.writes_cache and c >= i:
                raise ValueError(f"schedule[{i}] reads cache entry {c}, which has not run yet")
        for a in self.stream_adds:
            if not 0 <= a.before < len(self.schedule):
                raise ValueError(f"a stream addition names schedule entry {a.before}, outside the schedule")
            if a.table is not None and (a.table not in self.stream_tables
                                        or not 0 <= a.row < self.stream_tables[a.table][0]):
                raise ValueError(f"a stream addition names row {a.row} of '{a.table}', which the plan does not declare")
            if a.matrix is not None and (a.embedding or self.stream_matrices.get(a.matrix) != (self.hidden_size, 2 * self.hidden_size)):
                raise ValueError(f"a stream addition names the matrix '{a.matrix}', which the plan does not declare as "
                                 f"[hidden, 2 hidden] (or adds the embedding output beside it)")


@dataclass
class BuildEnv:
    """What parts need at build and run time besides their own parameters."""
    device: torch.device
    dtype: torch.dtype                 # activation / matrix dtype: float32 or bfloat16
    workspace: Any = None              # engine.workspace.Workspace
    # A norm split between two products (ops.kernels.SplitNorm), handed from a block to a part for
    # one call.  A part that sets `split_norm = True` takes `split_in` (its input rows are then
    # the split's values, and its first product scales by the split) and `split_out` (its last
    # adding product leaves the split's values and sums); the others never look at them.
    split_in: Any = None
    split_out: Any = None
    next_block_norm: Any = None        # the norm that reads the residual after this block (set by the model)

    def take_split_in(self):
        s, self.split_in = self.split_in, None
        return s

    def take_split_out(self):
        s, self.split_out = self.split_out, None
        return s

    @property
    def is_float32(self) -> bool:
        return self.dtype == torch.float32


class Part:
    split_norm = False     # True: forward() honours env.split_in / env.split_out (see BuildEnv)

    def split_reader_weight(self):
        """For parts with `split_norm`: the weight [N, K] of the product that reads the part's input
        (the one that gets `scale=`), so that a block offers a split only where that product can
        take it.  None: the block offers it only for steps the weight stream runs."""
        return None

    def tensors(self) -> dict[str, TensorSpec]:
        return {}

    def load(self, tensors: dict[str, torch.Tensor], env: BuildEnv) -> None:
        pass

    # ---- what a row costs, for reports (a roofline needs no knowledge of the architecture) ----
    def flops_per_row(self) -> int:
        """Floating-point operations of one row through the part's matrix products (2 per multiply-add)."""
        n = 0
        for spec in self.tensors().values():
            if spec.role == MATRIX:
                k = 1
                for d in spec.shape:
                    k *= int(d)
                n += 2 * k
        return n

    def unread_weight_bytes(self, rows: int) -> float:
        """Bytes of the part's weights that a step of `rows` rows is expected NOT to read (experts nobody chose)."""
        return 0.0


class Mixer(Part):
    def cache_spec(self) -> KVSpec | StateSpec | tuple | None:
        return None

    def forward(self, h, out, accumulate, batch, cache, env) -> None:
        raise NotImplementedError

    def flops_per_query_key(self) -> int:
        """Operations per (query row, cached position) pair, for mixers that look back over the sequence."""
        return 0


class FeedForward(Part):
    def forward(self, h, out, accumulate, batch, env) -> None:
        raise NotImplementedError


class PositionEncoding(Part):
    """How a mixer's queries and keys learn their positions.  A part either names a rotation the
    mixer's fused kernel can apply (`fused_rotary`), or encodes q and k itself (`apply`); the
    mixer asks in this order and knows nothing else about the encoding."""

    def fused_rotary(self):
        """(inverse frequencies [rope_dim/2] float or None for no rotation, rope_dim, split-half
        pairing?) when the encoding is a rotation by position * frequency; None otherwise."""
        return None

    def apply(self, q: torch.Tensor, k: torch.Tensor | None, row_pos: torch.Tensor) -> None:
        """Encodes in place: q [rows, heads, head_dim], k [rows, kv heads, head_dim] (None when the
        layer stores no keys), row_pos int32 [rows] absolute positions."""
        raise NotImplementedError
