"""What every part of a layer has in common: declared tensors and a build context.

A part is built from (a) its parameters, taken verbatim from a `PartSpec`,
(b) the tensors it declared, already on the device, and (c) a `BuildContext`
that carries the compute dtype, the device and the table of kernels.  A part
never sees a model config and never names an architecture.

Interfaces (duck-typed; the classes below only document them):

* Norm:          `forward(residual, delta=None, rows=None) -> Tensor`
                 adds `delta` into the fp32 `residual` (in place) and returns the
                 normalised rows in the compute dtype; with `rows`, only those
                 rows are produced and `residual` is left untouched.  `delta` is
                 what a mixer or feed-forward returned: [T, H], or float32
                 [splits, T, H] partial sums that the norm adds up in order.
* FeedForward:   `forward(x, batch) -> Tensor` of the same shape as `x`.
* Mixer:         `cache_needs() -> CacheNeeds`, and
                 `forward(x, batch, cache, owns_cache) -> Tensor`.
                 `cache` is the view the cache manager made for this run from
                 `cache_needs()`; `owns_cache` is False when the run reads
                 another run's cache and must not write it.
* PositionEncoding: `encode_and_store(qkv, geometry, batch, paged, write)`.
* Embedding:     `forward(batch) -> Tensor` float32 [T, H]: the residual stream's start, from
                 `batch.token_ids` (and whatever else of the batch it needs: positions, ...).
* Block arrangement: built as `cls(mixer, feed_forward, norms)` (`norms`: name -> norm; a
                 part the layer does not have is None), with a fourth argument `extras`
                 (name -> built layer extra) where the layer has some; `forward(residual,
                 pending, batch, cache, owns_cache)` returns the delta that the next norm has to
                 add (a tensor, or a `GatedDelta` / `NormedDelta` / `ScaledBranches` / `BranchSum`
                 for norms or arrangements that take one).  An arrangement
                 whose extras keep state per request answers `state_needs() -> StateNeeds`.
* Stream part:   `forward(residual, pending, start) -> float32 [T, H]`: the stream that replaces
                 `residual` in front of a run whose `RunSpec.remix` names the part; `pending` is
                 what the run before left to be added (or None), `start` the embedding's output.
                 A part that `RunSpec.average` names answers `behind(pending, start, results, index)
                 -> DepthAverage` instead.
* Layer extra:   whatever its arrangement calls; `declare(params)` and `__init__(params,
                 tensors, ctx)` like every part.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

import torch


@dataclass(frozen=True)
class TensorDecl:
    """A tensor that a part expects in the weight file."""

    name: str
    shape: tuple[int, ...]
    init: str = "normal"          # "normal" | "ones" | "zeros": used by the random-weights mode
    matrix: bool = True           # matrices feed GEMMs and are held in the compute dtype
    optional: bool = False        # the file may lack it; the part then finds no such name
    ignored: bool = False         # tolerated in the file (shape-checked) but never read: a
                                  # redundant copy, such as the head's matrix of a tied model


@dataclass
class BuildContext:
    dtype: torch.dtype            # compute dtype: torch.bfloat16 or torch.float32
    device: torch.device
    ops: Any                      # kernel table (ops.CudaOps on the product path)

    def place(self, t: torch.Tensor, *, matrix: bool) -> torch.Tensor:
        """Move a loaded tensor to the device in the precision it is held in.

        float32 compute: every floating tensor becomes float32.  bfloat16
        compute: matrices become bfloat16; other tensors keep the precision they
        were stored in (a tensor stored in 32-bit stays so); integer tensors
        become int32.
        """
        if not t.is_floating_point():
            return t.to(device=self.device, dtype=torch.int32).contiguous()
        if self.dtype == torch.float32:
            return t.to(device=self.device, dtype=torch.float32).contiguous()
        if matrix or t.dtype != torch.float32:
            return t.to(device=self.device, dtype=self.dtype).contiguous()
        return t.to(device=self.device).contiguous()


@dataclass(frozen=True)
class PagedKVNeeds:
    """Keys and values that grow with the sequence, kept in pages."""

    num_kv_heads: int
    head_dim: int                 # width of a key
    window: int | None = None     # None: all keys; n: only the last n positions are ever read
    value_dim: int | None = None  # width of a value; None: the same as a key's; 0: no values
                                  # are stored (the keys are read as values too)
    keep_first: int = 0           # beside a window: positions below this stay readable for good

    @property
    def value_width(self) -> int:
        return self.head_dim if self.value_dim is None else self.value_dim


@dataclass(frozen=True)
class StateNeeds:
    """Per-request state of fixed size: name -> (shape, dtype)."""

    tensors: Mapping[str, tuple[tuple[int, ...], torch.dtype]] = field(default_factory=dict)


@dataclass(frozen=True)
class CacheNeeds:
    paged: PagedKVNeeds | None = None
    state: StateNeeds | None = None


@dataclass
class GatedDelta:
    """What a gated residual branch hands to the next norm: the branch's result ([T, H], or
    float32 [splits, T, H] partial sums) and the gate's logits [T, H] (rows may lie further
    apart than H: a view into a wider product; or float32 partial sums as well).  The norm adds sigmoid(logits) * delta."""

    delta: torch.Tensor
    gate_logits: torch.Tensor | None = None


@dataclass
class NormedDelta:
    """What a branch with a norm of its own behind it hands to the next norm: the branch's result
    ([T, H], or float32 [splits, T, H] partial sums) and that norm's weight and eps.  The next
    norm adds rmsnorm(delta) * weight to the residual stream before it normalises."""

    delta: torch.Tensor
    weight: torch.Tensor
    eps: float


@dataclass
class ScaledBranches:
    """What a layer whose mixer and feed-forward read the same stream hands to the next norm: the
    two results (each [T, H] or float32 [splits, T, H] partial sums; the second may be absent),
    a per-channel scale for each (or None) and the factor of their sum.  The next norm adds
    mult * (scale_a * a + scale_b * b) to the residual stream before it normalises.  `extra`:
    float32 [T, H] rows that are added as well (see `with_extra_rows`)."""

    a: torch.Tensor
    scale_a: torch.Tensor | None
    b: torch.Tensor | None
    scale_b: torch.Tensor | None
    mult: float
    extra: torch.Tensor | None = None


@dataclass
class BranchSum:
    """What a layer whose mixer and feed-forward read the output of one norm hands to the next
    norm: the mixer's result ([T, H], or float32 [splits, T, H] partial sums) and the
    feed-forward's (float32 [T, H], or None for a layer without one).  The next norm adds
    both to the residual stream before it normalises."""

    a: torch.Tensor
    b: torch.Tensor | None = None


@dataclass
class StreamStart:
    """The stream begins as these float32 rows [T, H], which stay as they are: the first norm reads
    them and writes the stream (a schedule that needs the embedding's output later on)."""

    rows: torch.Tensor


@dataclass
class DepthAverage:
    """What a run behind which the stream is averaged over depth hands to the next norm: what is
    pending (None, a tensor or partial sums, or a `NormedDelta`), the embedding's output X_0
    (float32 [T, H]), the record of the runs' results (float32 [runs, T, H]: X_j lies at j - 1), this
    run's number n (from 1 on) and float32 coefficients [n + 1].  The next norm adds what is pending
    to the stream, which is the result X_n, stores it and replaces the stream by the sum over j of
    coefficient j times X_j before it goes on."""

    pending: Any
    start: torch.Tensor
    results: torch.Tensor
    n: int
    coefficients: torch.Tensor


def with_extra_rows(pending, rows: torch.Tensor):
    """`pending` with float32 rows [T, H] that the next norm adds to the residual stream as well
    (a schedule that adds the embedding's output again in front of a run).  Only what a norm can
    add in the same pass takes them."""
    if isinstance(pending, ScaledBranches):
        return ScaledBranches(pending.a, pending.scale_a, pending.b, pending.scale_b, pending.mult, rows)
    raise ValueError("the layer in front of a run that adds the embedding's output again must "
                     f"hand on its result as ScaledBranches, not {type(pending).__name__}")


def names_of(params: Mapping[str, Any]) -> Mapping[str, str]:
    names = params.get("names")
    if not isinstance(names, Mapping):
        raise ValueError("part parameters carry no 'names' mapping (logical -> tensor name)")
    return names
