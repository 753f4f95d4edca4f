"""The matrix memory of xLSTM (mLSTM): a recurrent mixer with a matrix state per head, exponential gates and a normalizer.

    q = W_q h * dim^-1/2, k = W_k h (``heads`` heads of ``dim``), v = W_v h (``heads`` heads of ``vdim``); one number per head each:
    log input gate i = cap tanh((W_i h + b_i) / cap), log forget gate f = logsigmoid(cap tanh((W_f h + b_f) / cap))
    per head, with S [dim, vdim], n [dim] and a running maximum m carried from token to token in float32, all 0 at the start:
        m' = max(f + m, i);   S <- exp(f + m - m') S + exp(i - m') k v^T;   n <- exp(f + m - m') n + exp(i - m') k;   m <- m'
        o = S^T q / (max(|<n, q>|, exp(-m)) + 1e-6)
    every head's o is divided by its root mean square over vdim; the heads are concatenated, multiplied by a weight of all heads'
    size and by sigmoid(W_g h), then projected by W_o

The recurrence runs on the kernels of csrc/kernels/gated_delta.cu: n is one more value channel of the state whose value is
always 1, so that the walk carries it like the others; the running maximum is scanned by a kernel of its own before the walk.

Kept per request: the state, per head dim rows of vdim numbers followed by the dim numbers of n, and the heads' running maxima, all
float32 in both precisions.  One product gives q | k | v | g | i | f in float32.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import ops
from .base import BundleCacheSpec, Mixer, Part, StateCacheSpec, TensorGetter, TensorSpec
from .linear import ACCUM, STORE_F32, Linear


class MatrixMemory(Mixer):
    graph_safe = True
    can_store = True

    def __init__(self, hidden: int, heads: int, dim: int, vdim: int, gate_cap: float, prefix: str, eps: float, gate: str = "sigmoid",
                 out_scale: float = 1.0):
        """Tensors ``prefix.q``, ``.k``, ``.v``, ``.g``, ``.i``, ``.f`` (+ ``.i.b``, ``.f.b`` [heads]), ``.norm`` [heads * vdim], ``.o``."""
        if gate not in ("silu", "sigmoid"):
            raise ValueError(f"gate '{gate}' (silu, sigmoid)")
        if not gate_cap > 0.0:
            raise ValueError(f"gate_cap {gate_cap} must be positive")
        self.hidden, self.heads, self.dim, self.vdim, self.gate_cap = hidden, heads, dim, vdim, float(gate_cap)
        self.prefix, self.eps, self.gate, self.out_scale = prefix, float(eps), gate, float(out_scale)
        p = prefix
        self.inp = Linear(hidden, [heads * dim, heads * dim, heads * vdim, heads * vdim, heads, heads],
                          [f"{p}.{t}" for t in ("q", "k", "v", "g", "i", "f")], pad_rows_to=4)
        self.o = Linear(heads * vdim, [hidden], [f"{p}.o"])
        self.gate_bias: Optional[torch.Tensor] = None    # float32 [2 heads]: input gates, then forget gates
        self.norm_w: Optional[torch.Tensor] = None       # float32 [heads * vdim]

    def children(self) -> List[Part]:
        return [self.inp, self.o]

    def tensor_specs(self) -> List[TensorSpec]:
        p, H = self.prefix, self.heads
        return [TensorSpec(f"{p}.i.b", (H,), "bias"), TensorSpec(f"{p}.f.b", (H,), "bias"), TensorSpec(f"{p}.norm", (H * self.vdim,), "norm")]

    def load(self, get: TensorGetter, device, dtype) -> None:
        f32 = lambda name: get(f"{self.prefix}.{name}").to(device).to(torch.float32).contiguous()
        self.gate_bias = torch.cat([f32("i.b"), f32("f.b")]).contiguous()
        self.norm_w = f32("norm")

    def cache_spec(self):
        return BundleCacheSpec(StateCacheSpec((self.heads, self.dim * (self.vdim + 1)), torch.float32),
                               (("maximum", StateCacheSpec((self.heads,), torch.float32)),))

    def step_bytes(self, tokens: int, element_size: int) -> int:
        H, d, dv = self.heads, self.dim, self.vdim
        prep = 2 * H * d + H * dv + 3 * H + 3
        return tokens * ((self.inp.padded_out + prep + H * (dv + 1)) * 4 + H * dv * element_size)

    def forward(self, ctx, h: torch.Tensor, x: torch.Tensor, cache, accumulate: bool = True) -> None:
        T = h.shape[0]
        H, d, dv = self.heads, self.dim, self.vdim
        proj = ctx.buffer((T, self.inp.padded_out), torch.float32)
        self.inp.forward(h, proj, STORE_F32)
        off_g = 2 * H * d + H * dv
        gz, gates = proj[:, off_g:off_g + H * dv], proj[:, off_g + H * dv:off_g + H * dv + 2 * H]
        prep = ctx.buffer((T, ops.gated_delta_prep_width(H, H, d, dv, ops.DECAY_EXP_GATES)), torch.float32)
        raw = ctx.buffer((T, H * (dv + 1)), torch.float32)
        out = ctx.buffer((T, H * dv))
        prof = ops.profiling()
        if prof is not None:
            prof.note_work(T * (2 * H * d + 2 * H * dv + 3 * H) * 4 + 2 * ctx.B * H * d * (dv + 1) * 4, 5 * T * H * d * (dv + 1))
        ops.gated_delta(proj, gates, gz, None, None, self.gate_bias, self.norm_w, prep, raw, cache.state, None, out,
                        ctx.seq_of_token, ctx.seq_slot, ctx.q_start, ctx.B, 0, 0, H, H, d, dv, 1, self.eps,
                        decay=ops.DECAY_EXP_GATES, gate=ops.GATE_SILU if self.gate == "silu" else ops.GATE_SIGMOID, delta=False,
                        out_scale=self.out_scale, operands=ops.OPERANDS_PLAIN, m_state=cache.extra["maximum"], cap=self.gate_cap,
                        normalizer=True)
        self.o.forward(out, x, ACCUM if accumulate else STORE_F32)
