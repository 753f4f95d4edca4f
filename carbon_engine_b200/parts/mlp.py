"""Gated feed-forward: down(act(gate(h)) * up(h)), added into the residual stream
(src/model/layers.rs:568, 625-648; src/model/mod.rs:649).  The activation is SiLU or ReLU; the gate and up
weights are held as one matrix so that one product with a gated epilogue serves both.  A third activation, "clamped", cuts both
values first: g = min(gate, limit), u = up within [-limit, limit], g sigmoid(alpha g) (u + 1).  It may come with biases on all
three projections: the gate's and the up's are added in the product's epilogue.
Dense feed-forward without a gate: down(act(up(h))), act the square of ReLU, the up product's epilogue."""
from __future__ import annotations

from typing import List, Optional, Sequence

import torch

from .base import FeedForward, Part
from .. import ops
from .linear import ACCUM, CLAMPGLU, RELU2, RELUGLU, STORE_F32, SWIGLU, Linear

_EPILOGUES = {"silu": SWIGLU, "relu": RELUGLU, "clamped": CLAMPGLU}


class GatedMLP(FeedForward):
    can_store = True

    def __init__(self, hidden: int, intermediate: int, prefix: str, activation: str = "silu",
                 names: Sequence[str] = ("gate_proj.weight", "up_proj.weight", "down_proj.weight"),
                 bias_names: Optional[Sequence[str]] = None, limit: float = 0.0, alpha: float = 1.0):
        """``names``: the gate, up and down tensors' names under ``prefix``; ``bias_names``: their biases' (with the clamped
        activation), or None.  ``limit``, ``alpha``: the clamped activation's constants."""
        if activation not in _EPILOGUES:
            raise ValueError(f"activation '{activation}' is not supported ({', '.join(sorted(_EPILOGUES))})")
        self.epilogue = _EPILOGUES[activation]
        self.hidden, self.intermediate, self.prefix = hidden, intermediate, prefix
        if bias_names is not None and activation != "clamped":
            raise ValueError("biases in front of the gate come with the clamped activation only")
        if activation == "clamped" and not limit > 0.0:
            raise ValueError(f"the clamped activation needs a positive limit, got {limit}")
        self.limit, self.alpha = float(limit), float(alpha)
        gate, up, down = names
        biases = [f"{prefix}.{b}" for b in bias_names] if bias_names is not None else [None] * 3
        self.gate_up = Linear(hidden, [intermediate, intermediate], [f"{prefix}.{gate}", f"{prefix}.{up}"], bias_names=biases[:2])
        self.down = Linear(intermediate, [hidden], [f"{prefix}.{down}"], bias_names=biases[2:])

    def children(self) -> List[Part]:
        return [self.gate_up, self.down]

    def step_bytes(self, tokens: int, element_size: int) -> int:
        return tokens * self.intermediate * element_size

    def forward(self, ctx, h: torch.Tensor, x: torch.Tensor, accumulate: bool = True):
        """With ``accumulate=False`` the down projection's bias, where there is one, is owed (returned)."""
        act = ctx.buffer((h.shape[0], self.intermediate))
        glu = ops.GluParams(self.limit, self.alpha, self.gate_up.bias) if self.epilogue == CLAMPGLU else None
        self.gate_up.forward(h, act, self.epilogue, glu=glu)
        self.down.forward(act, x, ACCUM if accumulate else STORE_F32, add_bias=accumulate)
        return None if accumulate else self.down.bias


class DenseMLP(FeedForward):
    """down(act(up(h))) with act = relu(z)^2 (``activation`` "relu2")."""
    can_store = True
    _ACTS = {"relu2": RELU2}

    def __init__(self, hidden: int, intermediate: int, prefix: str, activation: str = "relu2", names: Sequence[str] = ("up", "down")):
        if activation not in self._ACTS:
            raise ValueError(f"activation '{activation}' is not supported ({', '.join(sorted(self._ACTS))})")
        self.epilogue = self._ACTS[activation]
        self.hidden, self.intermediate, self.prefix = hidden, intermediate, prefix
        up, down = names
        self.up = Linear(hidden, [intermediate], [f"{prefix}.{up}"])
        self.down = Linear(intermediate, [hidden], [f"{prefix}.{down}"])

    def children(self) -> List[Part]:
        return [self.up, self.down]

    def step_bytes(self, tokens: int, element_size: int) -> int:
        return tokens * self.intermediate * element_size

    def forward(self, ctx, h: torch.Tensor, x: torch.Tensor, accumulate: bool = True) -> None:
        act = ctx.buffer((h.shape[0], self.intermediate))
        self.up.forward(h, act, self.epilogue)
        self.down.forward(act, x, ACCUM if accumulate else STORE_F32)
