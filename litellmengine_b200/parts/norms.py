"""Normalisation parts."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..config.specs import NormSpec
from ..csrc import ops
from ..weights.loader import ParamSpec
from .registry import register_norm


@register_norm("rmsnorm")
class RMSNorm:
    """out = v * rsqrt(mean(v^2) + eps) * weight with v = x (+ delta), everything in 32-bit
    (src/layers/rms_norm.cu:77-93).  The weight multiplies directly (no 1 + w).  `delta` may be a `PendingNormed`: a
    sublayer's output and the norm of this kind that it passes before it joins the stream, which the same kernel
    applies, with whatever else joins there; the sum is then written back into x unless `rows` picks rows."""

    accepts_partials = True    # `delta` may be an ops.PartialSum: the kernel adds the k-splits as it reads
    accepts_join = True        # and a PendingNormed with a `join`
    center = False             # what a kernel that applies this norm itself needs to know beside weight and eps

    def __init__(self, spec: NormSpec, size: int):
        self.eps = float(spec.eps)
        self.size = size
        self.name = getattr(spec, "weight_name", "weight")     # '' when the tensor is named like the norm itself
        self.weight: Optional[torch.Tensor] = None

    def parameters(self) -> Dict[str, ParamSpec]:
        return {self.name: ParamSpec((self.size,), role="scale", init=("one_plus_normal", 0.01))}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight = tensors[self.name].contiguous()

    def scale_output(self, factor) -> None:
        """From now on the norm's output is multiplied by `factor` (a number, or float32 [size]): it joins the weight."""
        self.weight = (self.weight * factor).contiguous()

    def add_normed(self, h: torch.Tensor, y, copy_dtype: Optional[torch.dtype] = None) -> Optional[torch.Tensor]:
        """h += norm(y) * weight in place (the norm of a sublayer's OUTPUT joined with the residual add);
        returns the new h in `copy_dtype` if one is asked for."""
        return ops.rmsnorm_add(h, y, self.weight, self.eps, copy_dtype)

    def forward(self, x: torch.Tensor, out_dtype: torch.dtype, delta: Optional[torch.Tensor] = None,
                rows: Optional[torch.Tensor] = None, write_sum: bool = False) -> torch.Tensor:
        if isinstance(delta, PendingNormed):
            y = delta.y
            if isinstance(y, ops.PartialSum) and y.rounds_to is not None:
                y = ops.as_tensor(y)                 # k-splits of a product that is not 32-bit: their sum is rounded first
            post = (delta.norm.weight, delta.norm.eps) if delta.norm is not None else None
            return ops.rmsnorm_sandwich(x, y, post, (self.weight, self.eps), out_dtype, rows=rows, join=delta.join)
        return ops.rmsnorm(x, self.weight, self.eps, out_dtype, delta=delta, rows=rows, write_sum=write_sum)


@register_norm("layernorm")
class LayerNorm:
    """out = (v - mean(v)) * rsqrt(mean((v - mean(v))^2) + eps) * weight (+ bias, when the spec has one: tensor 'b' beside
    the weight) with v = x (+ delta), everything in 32-bit.  The kernel is the one that serves models with several
    residual streams, run on one stream with unit coefficients.  `delta` may be a `PendingSum` or a `PendingStart`."""

    accepts_partials = True
    accepts_pending = True     # `delta` may be a PendingSum or a PendingStart
    center = True

    def __init__(self, spec: NormSpec, size: int):
        self.eps = float(spec.eps)
        self.size = size
        self.name = getattr(spec, "weight_name", "weight")
        self.has_bias = bool(getattr(spec, "bias", False))
        self.weight: Optional[torch.Tensor] = None
        self.bias: Optional[torch.Tensor] = None

    def parameters(self) -> Dict[str, ParamSpec]:
        p = {self.name: ParamSpec((self.size,), role="scale", init=("one_plus_normal", 0.01))}
        if self.has_bias:
            p["b"] = ParamSpec((self.size,), role="scale", init=("normal", 0.01))
        return p

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight = tensors[self.name].contiguous()
        if self.has_bias:
            self.bias = tensors["b"].contiguous()

    def forward(self, x: torch.Tensor, out_dtype: torch.dtype, delta=None, rows: Optional[torch.Tensor] = None,
                write_sum: bool = False) -> torch.Tensor:
        y2 = source = add = None
        if isinstance(delta, PendingStart):
            source, add, delta = delta.source, delta.add, delta.y
        elif isinstance(delta, PendingSum):
            delta, y2 = delta.y, delta.y2
        if isinstance(delta, ops.PartialSum) and delta.rounds_to is not None:
            delta = ops.as_tensor(delta)
        return ops.stream_norm(x, delta, None, None, None, self.weight, self.eps, True, out_dtype, rows=rows,
                               write_back=write_sum, bias=self.bias, y2=y2, source=source, add=add)


class PendingSum:
    """Two sublayer outputs that have not joined the residual stream yet (float32 tensors or `ops.PartialSum`s of float32
    products): the kernel that norms the next layer's input adds both as it reads."""

    def __init__(self, y, y2):
        self.y, self.y2 = y, y2

    @staticmethod
    def of(y, y2):
        """y + y2 as something a norm with `accepts_pending` takes as its delta; either may be None (already added)."""
        whole = lambda v: ops.as_tensor(v) if isinstance(v, ops.PartialSum) and v.rounds_to is not None else v
        y, y2 = whole(y), whole(y2)
        if y is None or y2 is None:
            return y if y2 is None else y2
        return PendingSum(y, y2)

    def settled(self) -> torch.Tensor:
        return ops.as_tensor(self.y) + ops.as_tensor(self.y2)


class PendingStart:
    """A stream that is about to be replaced: source + add (one row for all tokens) + y is the new stream, which the
    first norm of a pass makes and writes as it reads."""

    def __init__(self, source: torch.Tensor, add: torch.Tensor, y):
        self.source, self.add, self.y = source, add, y

    def settle_into(self, h: torch.Tensor) -> None:
        """For a norm that does not take it: write the new stream into h."""
        ops.stream_norm(h, self.y, None, None, None, None, 0.0, False, None, source=self.source, add=self.add)


class PendingNormed:
    """A sublayer's output that has not joined the residual stream yet, with the norm it passes on its way there
    (None: it joins as it is).  The kernel that norms the next sublayer's input applies both on the way.  `join`
    (float32, the stream's shape): one more summand that joins there, for norms with `accepts_join`."""

    def __init__(self, y, norm=None, join: Optional[torch.Tensor] = None):
        self.y, self.norm, self.join = y, norm, join


@register_norm("tanh")
class TanhNorm:
    """out = tanh(alpha * v) * weight + bias with v = x (+ what is pending), elementwise, everything in 32-bit: a norm
    that computes no mean and no variance (the spec's eps is not used).  `alpha` is one learned number.  Tensors:
    the weight under the norm's own name (or `weight_name`), `alpha` [] and `b` [size] beside it.  `delta` may be a
    `PendingNormed`: a sublayer's output and the norm of this kind that it passes before the residual add, which
    the same kernel applies; with `write_sum` (or always for a `PendingNormed`) the sum is written back into x."""

    accepts_partials = True
    center = False

    def __init__(self, spec: NormSpec, size: int):
        self.eps = float(spec.eps)
        self.size = size
        self.name = getattr(spec, "weight_name", "weight")
        self.weight = self.alpha = self.bias = None

    def parameters(self) -> Dict[str, ParamSpec]:
        return {self.name: ParamSpec((self.size,), role="scale", init=("one_plus_normal", 0.05)),
                "alpha": ParamSpec((), role="scale", init=("one_plus_normal", 0.1)),
                "b": ParamSpec((self.size,), role="scale", init=("normal", 0.05))}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight = tensors[self.name].contiguous()
        self.alpha = tensors["alpha"].reshape(1).contiguous()
        self.bias = tensors["b"].contiguous()

    def triple(self):
        return (self.alpha, self.weight, self.bias)

    def forward(self, x: torch.Tensor, out_dtype: torch.dtype, delta=None, rows: Optional[torch.Tensor] = None,
                write_sum: bool = False) -> torch.Tensor:
        post = None
        if isinstance(delta, PendingNormed):
            post = delta.norm.triple() if delta.norm is not None else None
            delta = delta.y
        if isinstance(delta, ops.PartialSum) and delta.rounds_to is not None:
            delta = ops.as_tensor(delta)             # k-splits of a product that is not 32-bit: their sum is rounded first
        return ops.tanh_norm(x, delta, post, self.triple(), out_dtype, rows=rows)

    def add_normed(self, h: torch.Tensor, y) -> None:
        """h += norm(y) in place, nothing returned: the norm on a sublayer's output with nothing behind it."""
        ops.tanh_norm(h, y, self.triple(), None)
