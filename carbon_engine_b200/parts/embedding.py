"""Token embedding and the language-model head.

x0[t] = E[token[t]], no scaling (src/model/mod.rs:781-784).  The head takes the final norm of the
requested rows only and multiplies by the head matrix into float32 logits
(src/model/mod.rs:793-802); with tied embeddings the head IS the embedding tensor
(src/model/mod.rs:735): the same memory, no copy.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import ops
from .base import RESIDUAL_ROUNDED, Norm, Part, TensorGetter, TensorSpec, to_device
from .linear import STORE_F32, matmul_nt
from .norm import RMSNorm


class Embedding(Part):
    def __init__(self, vocab: int, width: int, name: str, scale: float = 1.0, norm: Optional[RMSNorm] = None,
                 leave_rounded: bool = False):
        """``scale`` multiplies every embedding row on its way into the residual stream; ``norm`` is taken of it then (in the same
        kernel).  ``leave_rounded``, with a norm: the first block reads the residual itself, and finds it rounded."""
        self.vocab, self.width, self.name, self.scale = vocab, width, name, float(scale)
        self.norm, self.leave_rounded = norm, bool(leave_rounded)
        self.weight: Optional[torch.Tensor] = None

    def tensor_specs(self) -> List[TensorSpec]:
        return [TensorSpec(self.name, (self.vocab, self.width), "embedding")]

    def children(self) -> List[Part]:
        return [self.norm] if self.norm is not None else []

    def load(self, get: TensorGetter, device, dtype) -> None:
        self.weight = to_device(get(self.name), device, dtype)

    def forward(self, ctx, x: torch.Tensor) -> None:
        if self.norm is not None:
            rounded = ctx.buffer(tuple(x.shape)) if self.leave_rounded and ctx.dtype == torch.bfloat16 else None
            ops.embed_norm(self.weight, ctx.tokens, self.norm.weight, x, ctx.status, self.norm.eps, self.scale, rounded)
            if rounded is not None:
                ctx.shared[RESIDUAL_ROUNDED] = (rounded, x.data_ptr())
            return
        ops.embed(self.weight, ctx.tokens, x, ctx.status, self.scale)


class LMHead(Part):
    """Final norm + head product for chosen rows.  ``tied_to`` shares an embedding's tensor."""

    def __init__(self, vocab: int, width: int, norm: Norm, name: Optional[str], tied_to: Optional[Embedding] = None,
                 redundant_name: Optional[str] = None, logit_cap: float = 0.0):
        """``logit_cap`` > 0: the logits become cap * tanh(logits / cap).  ``redundant_name``: with a tied head, the name under which a checkpoint may still store a copy
        of the head; it is ignored, as the reference ignores it (src/model/mod.rs:725)."""
        if (name is None) == (tied_to is None):
            raise ValueError("the head has either a tensor of its own or an embedding it is tied to")
        self.vocab, self.width, self.norm, self.name, self.tied_to = vocab, width, norm, name, tied_to
        self.redundant_name = redundant_name if tied_to is not None else None
        self.logit_cap = float(logit_cap)
        self._weight: Optional[torch.Tensor] = None

    def ignorable_tensors(self) -> List[str]:
        return [self.redundant_name] if self.redundant_name else []

    def children(self) -> List[Part]:
        return [self.norm]

    def tensor_specs(self) -> List[TensorSpec]:
        return [] if self.name is None else [TensorSpec(self.name, (self.vocab, self.width), "linear")]

    def load(self, get: TensorGetter, device, dtype) -> None:
        if self.name is not None:
            self._weight = to_device(get(self.name), device, dtype)

    @property
    def weight(self) -> torch.Tensor:
        return self.tied_to.weight if self.tied_to is not None else self._weight

    def forward(self, ctx, x: torch.Tensor, rows: torch.Tensor) -> torch.Tensor:
        R = rows.shape[0]
        logits = torch.empty((R, self.vocab), dtype=torch.float32, device=x.device)
        if R == 0:
            return logits
        z = ctx.buffer((R, self.width))
        self.norm.forward(x, z, rows)
        matmul_nt(z, self.weight, logits, STORE_F32)
        if self.logit_cap > 0.0:
            ops.tanh_cap(logits, self.logit_cap)
        return logits
