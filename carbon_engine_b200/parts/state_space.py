"""State-space duality (Mamba-2): a recurrent mixer with a matrix state per head, one decay per head and a step size.

    W_in h = [z: heads * vdim | x: heads * vdim | B: groups * state | C: groups * state | dt: heads]
    x, B and C pass a short causal convolution over time per channel (``taps`` taps, a bias, zeros before the sequence's
    start) and SiLU;  dt <- softplus(dt + dt_bias)
    per head (head h reads group h // (heads / groups)), with S [state, vdim] carried from token to token in float32:
        S <- exp(-exp(A_log_h) dt) S + dt B x^T;      y = S^T C + D_h x
    y <- y * silu(z), then divided by its root mean square in ``norm_groups`` equal parts of all heads' values, times a weight
    output = W_o y

The recurrence is the plain decaying sum of outer products of csrc/kernels/gated_delta.cu with C as the query, B as the key, x as
the value and dt as what the written value is multiplied by; the gate comes before the norm in its finish.

Kept per request: the state [heads, state, vdim] and the convolution's last ``taps - 1`` inputs, both float32 in both
precisions.  One product gives all inputs in float32; its rows are held as [C | B | x | z | dt], the order in which the kernels
read query, key and value.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import ops
from .base import BundleCacheSpec, Mixer, Part, StateCacheSpec, TensorGetter, TensorSpec, register_init_kind
from .linear import ACCUM, STORE_F32, Linear

register_init_kind("conv_taps", 0.0, 0.5, True)
register_init_kind("decay_log", 0.0, 0.5, True)
register_init_kind("skip", 1.0, 0.3, True)


class StateSpace(Mixer):
    graph_safe = True
    can_store = True

    def __init__(self, hidden: int, heads: int, vdim: int, state: int, groups: int, taps: int, prefix: str, eps: float,
                 norm_groups: int = 1, gate: str = "silu", out_scale: float = 1.0):
        """Tensors ``prefix.in``, ``.conv`` [channels, taps], ``.conv.b``, ``.dt_bias``, ``.A_log``, ``.D`` [heads], ``.norm``
        [heads * vdim], ``.o``."""
        if heads % groups:
            raise ValueError(f"{heads} heads are not a multiple of {groups} groups")
        if taps < 1:
            raise ValueError("the convolution needs at least one tap")
        if (heads * vdim) % norm_groups:
            raise ValueError(f"{heads * vdim} values cannot be normalised in {norm_groups} equal parts")
        if gate not in ("silu", "sigmoid"):
            raise ValueError(f"gate '{gate}' (silu, sigmoid)")
        self.hidden, self.heads, self.vdim, self.state, self.groups, self.taps = hidden, heads, vdim, state, groups, int(taps)
        self.prefix, self.eps, self.norm_groups, self.gate, self.out_scale = prefix, float(eps), int(norm_groups), gate, float(out_scale)
        inner, bc = heads * vdim, groups * state
        self.inner = inner
        self.channels = inner + 2 * bc
        z, x, b, c, dt = 0, inner, 2 * inner, 2 * inner + bc, 2 * inner + 2 * bc
        total = dt + heads
        self.inp = Linear(hidden, [total], [f"{prefix}.in"], pad_rows_to=4,
                          row_order=[(c, dt), (b, c), (x, b), (z, x), (dt, total)])
        self.o = Linear(inner, [hidden], [f"{prefix}.o"])
        self.conv_w: Optional[torch.Tensor] = None       # [channels, taps] float32: C, B, x rows
        self.conv_b: Optional[torch.Tensor] = None       # [channels] float32
        self.a_log: Optional[torch.Tensor] = None
        self.dt_bias: Optional[torch.Tensor] = None
        self.skip: Optional[torch.Tensor] = None
        self.norm_w: Optional[torch.Tensor] = None

    def children(self) -> List[Part]:
        return [self.inp, self.o]

    def tensor_specs(self) -> List[TensorSpec]:
        p, H = self.prefix, self.heads
        return [TensorSpec(f"{p}.conv", (self.channels, self.taps), "conv_taps"), TensorSpec(f"{p}.conv.b", (self.channels,), "bias"),
                TensorSpec(f"{p}.dt_bias", (H,), "bias"), TensorSpec(f"{p}.A_log", (H,), "decay_log"), TensorSpec(f"{p}.D", (H,), "skip"),
                TensorSpec(f"{p}.norm", (self.inner,), "norm")]

    def load(self, get: TensorGetter, device, dtype) -> None:
        f32 = lambda name: get(f"{self.prefix}.{name}").to(device).to(torch.float32).contiguous()
        inner, bc = self.inner, self.groups * self.state
        order = lambda t: torch.cat([t[inner + bc:], t[inner:inner + bc], t[:inner]], dim=0).contiguous()      # x, B, C -> C, B, x
        self.conv_w, self.conv_b = order(f32("conv")), order(f32("conv.b"))
        self.a_log, self.dt_bias, self.skip, self.norm_w = f32("A_log"), f32("dt_bias"), f32("D"), f32("norm")

    def cache_spec(self):
        state = StateCacheSpec((self.heads, self.state, self.vdim), torch.float32)
        if self.taps == 1:
            return state
        return BundleCacheSpec(state, (("conv", StateCacheSpec((self.taps - 1, self.channels), torch.float32)),))

    def step_bytes(self, tokens: int, element_size: int) -> int:
        prep = self.channels + 2 * self.heads + 3
        return tokens * ((self.inp.padded_out + prep + self.inner) * 4 + self.inner * element_size)

    def forward(self, ctx, h: torch.Tensor, x: torch.Tensor, cache, accumulate: bool = True) -> None:
        T = h.shape[0]
        H, G, N, dv = self.heads, self.groups, self.state, self.vdim
        proj = ctx.buffer((T, self.inp.padded_out), torch.float32)
        self.inp.forward(h, proj, STORE_F32)
        off_z = self.channels
        gz, dec = proj[:, off_z:off_z + self.inner], proj[:, off_z + self.inner:off_z + self.inner + H]
        prep = ctx.buffer((T, ops.gated_delta_prep_width(H, G, N, dv, ops.DECAY_PER_HEAD)), torch.float32)
        raw = ctx.buffer((T, self.inner), torch.float32)
        out = ctx.buffer((T, self.inner))
        prof = ops.profiling()
        if prof is not None:         # what the walk reads and writes once, the state of every sequence twice
            prof.note_work(T * (2 * G * N + 2 * H * dv + 2 * H) * 4 + 2 * ctx.B * H * N * dv * 4, 5 * T * H * N * dv)
        kept = cache.extra["conv"] if self.taps > 1 else None
        ops.gated_delta(proj, dec, gz, self.conv_w, self.a_log, self.dt_bias, self.norm_w, prep, raw, cache.state, kept, out,
                        ctx.seq_of_token, ctx.seq_slot, ctx.q_start, ctx.B, 0, 0, H, G, N, dv, self.taps, self.eps,
                        decay=ops.DECAY_PER_HEAD, gate=ops.GATE_SILU if self.gate == "silu" else ops.GATE_SIGMOID, delta=False,
                        out_scale=self.out_scale, operands=ops.OPERANDS_CONV, conv_bias=self.conv_b, write_step=True, skip=self.skip,
                        norm_parts=self.norm_groups)
        self.o.forward(out, x, ACCUM if accumulate else STORE_F32)
