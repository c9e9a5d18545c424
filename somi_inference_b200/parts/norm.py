"""RMS normalisation over the last dimension, fused with the residual sum.

Formula (somi_inference/models/qwen2.py:46-62): x32 = float(x);
y = x32 * rsqrt(mean(x32^2) + eps); out = weight * y.  The reference casts y to
the input dtype before the weight multiply; here the residual stream stays in
float32 and the product is rounded once, at the end.
"""

from __future__ import annotations

import torch

from .base import (BranchSum, BuildContext, DepthAverage, GatedDelta, NormedDelta, ScaledBranches,
                   StreamStart, TensorDecl, names_of)
from .registry import NORMS


def update_stream(ops, residual: torch.Tensor, delta, weight, eps: float, out, rows=None) -> None:
    """Bring `residual` up to date with `delta` (None, a tensor, partial sums, a `NormedDelta`, a
    `StreamStart` or a `DepthAverage` of one of the former) and write it to `out` (where given), as it
    is or RMS-normed with `weight`, in one kernel.  With `rows` only those rows of `out` are made."""
    average, x_in = None, residual
    if isinstance(delta, DepthAverage):
        average = (delta.start, delta.results, delta.n, delta.coefficients)
        delta = delta.pending
    if isinstance(delta, StreamStart):
        x_in, delta = delta.rows, None
    weight_b, eps_b = None, 0.0
    if isinstance(delta, NormedDelta):
        delta, weight_b, eps_b = delta.delta, delta.weight, delta.eps
    if delta is not None and not isinstance(delta, torch.Tensor):
        raise ValueError(f"the stream cannot take up a {type(delta).__name__} here")
    ops.stream_update(x_in, None if rows is not None else residual, delta, weight_b, eps_b, average,
                      weight, eps, out, rows)


@NORMS.register("rmsnorm")
class RMSNorm:
    """`offset` (0 where not given): the weight is stored as what the factor exceeds it by, so the
    factor is offset + weight."""

    @staticmethod
    def declare(params) -> list[TensorDecl]:
        return [TensorDecl(names_of(params)["weight"], (int(params["size"]),),
                           init="zeros" if params.get("offset") else "ones", matrix=False)]

    def __init__(self, params, tensors, ctx: BuildContext) -> None:
        self.size = int(params["size"])
        self.eps = float(params["eps"])
        self.ctx = ctx
        self.weight = tensors[names_of(params)["weight"]]
        if params.get("offset"):
            self.weight = (float(params["offset"]) + self.weight.float()).contiguous()

    def forward(self, residual: torch.Tensor, delta: torch.Tensor | None = None,
                rows: torch.Tensor | None = None) -> torch.Tensor:
        """`delta` is [T, size], or float32 [splits, T, size] partial sums that are added up; or a
        `NormedDelta`: the branch's result passes an RMS norm of its own before it is added; or a
        `StreamStart` or `DepthAverage` (see `update_stream`)."""
        n = residual.shape[0] if rows is None else rows.shape[0]
        out = torch.empty((n, self.size), dtype=self.ctx.dtype, device=residual.device)
        if isinstance(delta, BranchSum):
            delta = ScaledBranches(delta.a, None, delta.b, None, 1.0)
        if isinstance(delta, ScaledBranches):
            self.ctx.ops.add_scaled_rmsnorm(residual, delta.a, delta.scale_a, delta.b, delta.scale_b,
                                            delta.mult, delta.extra, self.weight, None, self.eps,
                                            out, None, rows)
        elif isinstance(delta, (StreamStart, DepthAverage)):
            update_stream(self.ctx.ops, residual, delta, self.weight, self.eps, out, rows)
        elif isinstance(delta, NormedDelta):
            self.ctx.ops.add_normed_rmsnorm(residual, delta.delta, delta.weight, delta.eps,
                                            self.weight, self.eps, out, rows)
        else:
            self.ctx.ops.add_rmsnorm(residual, delta, self.weight, self.eps, out, rows)
        return out

    def forward_pair(self, residual: torch.Tensor, delta, other: "RMSNorm | None"):
        """Add `delta` (a `ScaledBranches`, a tensor, partial sums or None) to the residual
        stream and normalise it twice, with this norm's weight and with `other`'s (None: once),
        in one pass over the rows.  Returns the two results (the second None without `other`)."""
        if delta is not None and not isinstance(delta, ScaledBranches):
            if isinstance(delta, (NormedDelta, GatedDelta)):
                raise ValueError("a layer of parallel branches cannot follow one whose result "
                                 "passes a norm or a gate of its own")
            delta = ScaledBranches(delta, None, None, None, 1.0)
        if other is not None and other.weight.dtype != self.weight.dtype:
            raise ValueError("the two norms of a layer hold their weights in one precision")
        shape = (residual.shape[0], self.size)
        out1 = torch.empty(shape, dtype=self.ctx.dtype, device=residual.device)
        out2 = None if other is None else torch.empty(shape, dtype=self.ctx.dtype, device=residual.device)
        d = delta
        self.ctx.ops.add_scaled_rmsnorm(
            residual, None if d is None else d.a, None if d is None else d.scale_a,
            None if d is None else d.b, None if d is None else d.scale_b,
            1.0 if d is None else d.mult, None if d is None else d.extra, self.weight,
            None if other is None else other.weight, self.eps, out1, out2, None)
        return out1, out2


@NORMS.register("none")
class NoNorm:
    """Not a norm but what stands in its place where a sublayer reads the stream itself: brings the
    stream up to date with what is pending (see `update_stream`) and returns its rows in the
    compute dtype (float32 compute: the stream itself, which the next norm changes)."""

    @staticmethod
    def declare(params) -> list[TensorDecl]:
        return []

    def __init__(self, params, tensors, ctx: BuildContext) -> None:
        self.size = int(params["size"])
        self.ctx = ctx

    def forward(self, residual: torch.Tensor, delta=None, rows: torch.Tensor | None = None) -> torch.Tensor:
        if rows is None and self.ctx.dtype == torch.float32:
            if delta is not None:
                update_stream(self.ctx.ops, residual, delta, None, 0.0, None)
            return residual
        n = residual.shape[0] if rows is None else rows.shape[0]
        out = torch.empty((n, self.size), dtype=self.ctx.dtype, device=residual.device)
        update_stream(self.ctx.ops, residual, delta, None, 0.0, out, rows)
        return out


@NORMS.register("layernorm")
class LayerNorm:
    """(x - mean) / sqrt(var + eps) * weight, var the mean of the squared deviations; plus a bias
    where `names` has one.  Mean, variance and the residual sum are float32.  `delta` may be a `GatedDelta`:
    the branch's result is then multiplied by sigmoid(gate logits) as it is added; or a
    `BranchSum`: both results of the layer before are added."""

    @staticmethod
    def declare(params) -> list[TensorDecl]:
        n, shape = names_of(params), (int(params["size"]),)
        decl = [TensorDecl(n["weight"], shape, init="ones", matrix=False)]
        if "bias" in n:
            decl.append(TensorDecl(n["bias"], shape, init="zeros", matrix=False))
        return decl

    def __init__(self, params, tensors, ctx: BuildContext) -> None:
        n = names_of(params)
        self.size = int(params["size"])
        self.eps = float(params["eps"])
        self.ctx = ctx
        self.weight = tensors[n["weight"]]
        self.bias = tensors[n["bias"]].to(self.weight.dtype) if "bias" in n else None

    def forward(self, residual: torch.Tensor, delta=None,
                rows: torch.Tensor | None = None) -> torch.Tensor:
        gate = extra = None
        if isinstance(delta, GatedDelta):
            delta, gate = delta.delta, delta.gate_logits
        elif isinstance(delta, BranchSum):
            delta, extra = delta.a, delta.b
            if extra is not None and extra.dtype != torch.float32:
                extra = extra.float()
        n = residual.shape[0] if rows is None else rows.shape[0]
        out = torch.empty((n, self.size), dtype=self.ctx.dtype, device=residual.device)
        self.ctx.ops.add_layernorm(residual, delta, gate, self.weight, self.eps, out, rows,
                                   extra=extra, bias=self.bias)
        return out
