"""The start of a pass of a looped span of layers: the stream is joined with the model's embedding output."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..config.specs import RejoinSpec
from ..csrc import ops
from ..weights.loader import ParamSpec
from .norms import PendingNormed, PendingStart, PendingSum


class EmbeddingRejoin:
    """In front of pass t the stream x becomes W [x; x0] + step[t] with x0 the embedding output, W [hidden, 2 hidden] and
    step [passes, hidden].  The half of W that reads x0 is applied once a step (`begin`), in 32-bit accumulators that are
    never rounded; `start` applies the other half to the stream and leaves the sum to the first norm of the pass, which
    adds as it reads (`PendingStart`)."""

    def __init__(self, spec: RejoinSpec, hidden_size: int, compute_dtype: torch.dtype):
        self.spec, self.hidden, self.dtype = spec, hidden_size, compute_dtype
        self.w_x = self.w_e = self.step = None

    def matrices(self):
        return [self.w_x, self.w_e]

    def parameters(self) -> Dict[str, ParamSpec]:
        return {self.spec.in_name: ParamSpec((self.hidden, 2 * self.hidden)),
                self.spec.step_name: ParamSpec((self.spec.passes, self.hidden), role="scale", init=("normal", 0.02))}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        w = tensors[self.spec.in_name]
        self.w_x, self.w_e = w[:, :self.hidden].contiguous(), w[:, self.hidden:].contiguous()
        self.step = tensors[self.spec.step_name].contiguous()
        ops.prepare_streaming(self.w_x)
        ops.prepare_streaming(self.w_e)

    def begin(self, x0: torch.Tensor) -> torch.Tensor:
        """x0 in the compute dtype; float32 [T, hidden], what every pass starts from."""
        return ops.linear(x0, self.w_e, out_dtype=torch.float32)

    def start(self, h: torch.Tensor, copy: Optional[torch.Tensor], delta, base: torch.Tensor, t: int) -> PendingStart:
        """`copy`: h in the compute dtype when somebody has made it already (nothing is pending then)."""
        y2 = None
        if isinstance(delta, PendingSum):
            delta, y2 = delta.y, delta.y2
        if copy is None:
            if delta is None:
                copy = h if self.dtype == torch.float32 else h.to(self.dtype)
            else:
                copy = ops.stream_norm(h, delta, None, None, None, None, 0.0, False, self.dtype, write_back=False, y2=y2)
        return PendingStart(base, self.step[t], ops.linear(copy, self.w_x, out_dtype=torch.float32, partials_ok=True))


class AddedEmbedding:
    """In front of every pass but the first the embedding output x0 is added to the stream.  It has no tensors: the
    embedding kernel writes x0 twice, once as the stream, and the norm that makes the next sublayer's input adds it with
    the output that is still pending there (`PendingNormed.join`), or, in front of a norm that does not, the stream gets it
    in a kernel of its own."""

    def __init__(self, spec: RejoinSpec, hidden_size: int, compute_dtype: torch.dtype):
        self.spec = spec

    def matrices(self):
        return []

    def parameters(self) -> Dict[str, ParamSpec]:
        return {}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        pass

    def start(self, h: torch.Tensor, delta, x0: torch.Tensor, t: int, norm):
        """What is pending in front of `norm`, the first norm of pass t."""
        if t == 0:
            return delta
        if isinstance(delta, PendingNormed) and getattr(norm, "accepts_join", False):
            return PendingNormed(delta.y, delta.norm, join=x0)
        ops.residual_add(h, x0)                       # a sum: what is pending may join after it
        return delta


REJOINS = {"linear": EmbeddingRejoin, "add": AddedEmbedding}
