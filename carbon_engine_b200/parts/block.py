"""Arrangements of parts in a layer.  Pre-norm: x += mixer(norm1(x)); x += ffn(norm2(x))
(src/model/mod.rs:645-650).  Output-norm: x += norm1(mixer(x)); x += norm2(ffn(x)).  Sandwich-norm:
x += norm1b(mixer(norm1(x))); x += norm2b(ffn(norm2(x))).  Parallel: h = norm1(x); x += mixer(h) + ffn(h).
Post-norm: x <- norm1(alpha x + mixer(x)); x <- norm2(alpha x + ffn(x))."""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import ops
from .base import RESIDUAL_ROUNDED, Block, BundleCacheSpec, FeedForward, Mixer, Norm, Part
from .combine import NormedMixers
from .moe import RoutedExperts
from .norm import RMSNorm


def read_residual(ctx, x: torch.Tensor) -> torch.Tensor:
    """The residual as a sublayer's input: itself in float32, else its rounding, which the kernel that wrote it may have left."""
    if ctx.dtype == torch.float32:
        return x
    left = ctx.shared.pop(RESIDUAL_ROUNDED, None)
    if left is not None and left[1] == x.data_ptr() and left[0].shape == x.shape:
        return left[0]
    h = ctx.buffer(tuple(x.shape))
    ops.copy_cols(x, 0, x.shape[1], h)
    return h


class PreNormBlock(Block):
    def __init__(self, mixer_norm: Norm, mixer: Mixer, ffn_norm: Optional[Norm] = None, ffn: Optional[FeedForward] = None,
                 after: Optional[Part] = None):
        """``ffn`` None: the layer has only the mixer.  ``after``: a part with ``forward(ctx, x)`` that adds into the
        residual once the sublayers are done (a per-layer token input, for instance)."""
        if (ffn is None) != (ffn_norm is None):
            raise ValueError("a feed-forward and its norm come together")
        self.mixer_norm, self.mixer, self.ffn_norm, self.ffn, self.after = mixer_norm, mixer, ffn_norm, ffn, after

    def children(self) -> List[Part]:
        return [p for p in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn, self.after) if p is not None]

    def step_bytes(self, tokens: int, element_size: int) -> int:
        h = tokens * self.mixer_norm.width * element_size if hasattr(self.mixer_norm, "width") else 0
        parts = [self.mixer.step_bytes(tokens, element_size)]
        parts += [p.step_bytes(tokens, element_size) for p in (self.ffn, self.after) if p is not None]
        return h + max(parts)

    def forward(self, ctx, x: torch.Tensor, cache) -> None:
        h = ctx.buffer(tuple(x.shape))
        self.mixer_norm.forward(x, h)
        self.mixer.forward(ctx, h, x, cache)
        if self.ffn is not None:
            self.ffn_norm.forward(x, h)
            self.ffn.forward(ctx, h, x)
        if self.after is not None:
            self.after.forward(ctx, x)


class ParallelBlock(Block):
    """One norm, and both sublayers read its output: h = norm(x); x += mixer(h) + ffn(h).  ``ffn`` None: the layer has only the
    mixer.  Both sublayers add into the float32 residual, the mixer first."""

    def __init__(self, norm: Norm, mixer: Mixer, ffn: Optional[FeedForward] = None):
        self.norm, self.mixer, self.ffn = norm, mixer, ffn

    def children(self) -> List[Part]:
        return [p for p in (self.norm, self.mixer, self.ffn) if p is not None]

    def step_bytes(self, tokens: int, element_size: int) -> int:
        h = tokens * self.norm.width * element_size if hasattr(self.norm, "width") else 0
        ffn = self.ffn.step_bytes(tokens, element_size) if self.ffn is not None else 0
        return h + max(self.mixer.step_bytes(tokens, element_size), ffn)

    def forward(self, ctx, x: torch.Tensor, cache) -> None:
        h = ctx.buffer(tuple(x.shape))
        self.norm.forward(x, h)
        self.mixer.forward(ctx, h, x, cache)
        if self.ffn is not None:
            self.ffn.forward(ctx, h, x)


class OutputNormBlock(Block):
    """The norm sits on each sublayer's OUTPUT: x += norm1(mixer(x)); x += norm2(ffn(x)).  The sublayers read the
    residual itself, rounded to the compute dtype (in float32 they read it in place).  The sublayers STORE their result
    in a float32 buffer (``can_store``), and the norm's kernel adds its normalised rows into the residual."""

    def __init__(self, width: int, mixer: Mixer, mixer_norm: Norm, ffn: Optional[FeedForward] = None, ffn_norm: Optional[Norm] = None):
        if (ffn is None) != (ffn_norm is None):
            raise ValueError("a feed-forward and its norm come together")
        for part in (mixer, ffn):
            if part is not None and not getattr(part, "can_store", False):
                raise ValueError(f"{type(part).__name__} cannot store its output, which a norm on the output needs")
        for norm in (mixer_norm, ffn_norm):
            if norm is not None and not hasattr(norm, "add_into"):
                raise ValueError(f"{type(norm).__name__} cannot add its output into the residual")
        self.width, self.mixer, self.mixer_norm, self.ffn, self.ffn_norm = int(width), mixer, mixer_norm, ffn, ffn_norm

    def children(self) -> List[Part]:
        return [p for p in (self.mixer, self.mixer_norm, self.ffn, self.ffn_norm) if p is not None]

    def step_bytes(self, tokens: int, element_size: int) -> int:
        ffn = self.ffn.step_bytes(tokens, element_size) if self.ffn is not None else 0
        return tokens * self.width * (element_size + 4) + max(self.mixer.step_bytes(tokens, element_size), ffn)

    def _add(self, ctx, norm: Norm, y: torch.Tensor, x: torch.Tensor) -> None:
        """x += norm(y); in bfloat16 the norm's kernel also leaves the new residual rounded for the sublayer that reads it
        next (this block's feed-forward, or the next block's mixer)."""
        if ctx.dtype != torch.bfloat16:
            norm.add_into(y, x)
            return
        h = ctx.buffer(tuple(x.shape))
        norm.add_into(y, x, rounded=h)
        ctx.shared[RESIDUAL_ROUNDED] = (h, x.data_ptr())

    def forward(self, ctx, x: torch.Tensor, cache) -> None:
        y = ctx.buffer(tuple(x.shape), torch.float32)
        owed = self.mixer.forward(ctx, read_residual(ctx, x), y, cache, accumulate=False)
        if owed is not None:
            ops.add_bias(y, owed)
        self._add(ctx, self.mixer_norm, y, x)
        if self.ffn is None:
            return
        owed = self.ffn.forward(ctx, read_residual(ctx, x), y, accumulate=False)
        if owed is not None:
            ops.add_bias(y, owed)
        self._add(ctx, self.ffn_norm, y, x)


class PostNormBlock(Block):
    """The norm is taken of the weighted residual plus the sublayer's output, and IS the new residual: x <- mixer_norm(alpha x +
    mixer(x)); x <- ffn_norm(alpha x + ffn(x)).  The sublayers read the residual itself (rounded to the compute dtype) and STORE
    their result in a float32 buffer (``can_store``); one kernel weighs, adds and norms, and leaves the new residual rounded for
    the next sublayer.  The outputs of mixers side by side (:class:`NormedMixers`) are normed and added in that kernel too, and so
    are a token's experts (:class:`RoutedExperts` without a shared expert) summed.
    The norms are RMS norms.  ``ffn`` None: the layer has only the mixer."""

    def __init__(self, width: int, alpha: float, mixer: Mixer, mixer_norm: RMSNorm, ffn: Optional[FeedForward] = None,
                 ffn_norm: Optional[RMSNorm] = None):
        if (ffn is None) != (ffn_norm is None):
            raise ValueError("a feed-forward and its norm come together")
        for part in (mixer, ffn):
            if part is not None and not getattr(part, "can_store", False):
                raise ValueError(f"{type(part).__name__} cannot store its output, which a norm of the sum needs")
        for norm in (mixer_norm, ffn_norm):
            if norm is not None and not isinstance(norm, RMSNorm):
                raise ValueError(f"{type(norm).__name__}: this block's norms are RMS norms")
        self.width, self.alpha = int(width), float(alpha)
        self.mixer, self.mixer_norm, self.ffn, self.ffn_norm = mixer, mixer_norm, ffn, ffn_norm

    def children(self) -> List[Part]:
        return [p for p in (self.mixer, self.mixer_norm, self.ffn, self.ffn_norm) if p is not None]

    def step_bytes(self, tokens: int, element_size: int) -> int:
        ffn = self.ffn.step_bytes(tokens, element_size) if self.ffn is not None else 0
        return tokens * self.width * (2 * element_size + 4) + max(self.mixer.step_bytes(tokens, element_size), ffn)

    def _norm(self, ctx, x: torch.Tensor, outputs, norm: RMSNorm, picks=None, **more) -> None:
        rounded = ctx.buffer(tuple(x.shape)) if ctx.dtype == torch.bfloat16 else None
        if picks is not None:
            ops.residual_norm_picks(x, self.alpha, *picks, norm.weight, norm.eps, rounded)
        else:
            ops.residual_norm(x, self.alpha, outputs, norm.weight, norm.eps, rounded=rounded, **more)
        if rounded is not None:
            ctx.shared[RESIDUAL_ROUNDED] = (rounded, x.data_ptr())

    def forward(self, ctx, x: torch.Tensor, cache) -> None:
        h = read_residual(ctx, x)
        if isinstance(self.mixer, NormedMixers):
            m = self.mixer
            self._norm(ctx, x, m.outputs(ctx, h, cache), self.mixer_norm, member_weights=[n.weight for n in m.norms],
                       member_eps=m.norms[0].eps, factor=m.factor)
        else:
            y = ctx.buffer(tuple(x.shape), torch.float32)
            owed = self.mixer.forward(ctx, h, y, cache, accumulate=False)
            self._norm(ctx, x, [y], self.mixer_norm, bias=owed)
        if self.ffn is None:
            return
        h = read_residual(ctx, x)
        if isinstance(self.ffn, RoutedExperts) and self.ffn.shared_ff == 0:
            rows, pair_row, weights, _ = self.ffn.picks(ctx, h)
            self._norm(ctx, x, None, self.ffn_norm, picks=(rows, pair_row, weights))
            return
        y = ctx.buffer(tuple(x.shape), torch.float32)
        owed = self.ffn.forward(ctx, h, y, accumulate=False)
        self._norm(ctx, x, [y], self.ffn_norm, bias=owed)


class SandwichNormBlock(Block):
    """A norm in front of each sublayer and another on its OUTPUT: x += mixer_out(mixer(mixer_norm(x))); x += ffn_out(ffn(ffn_norm(x))).
    The sublayers STORE their result in a float32 buffer (``can_store``); one kernel adds the normed result (and a bias the
    sublayer still owes) into the residual and takes the norm that comes next: this block's ``ffn_norm``, or the norm in front of
    the next layer run (``ctx.next_norm``), whose block finds its input ready.  The norms are RMS norms.  ``ffn`` None: the layer has only the
    mixer."""

    #: what the last kernel left in ``ctx.shared``: (the norm it took, of which residual, its output)
    NORMED = "residual.normed"

    def __init__(self, width: int, mixer_norm: RMSNorm, mixer: Mixer, mixer_out: RMSNorm, ffn_norm: Optional[RMSNorm] = None,
                 ffn: Optional[FeedForward] = None, ffn_out: Optional[RMSNorm] = None):
        if len({ffn is None, ffn_norm is None, ffn_out is None}) != 1:
            raise ValueError("a feed-forward and its two norms come together")
        for part in (mixer, ffn):
            if part is not None and not getattr(part, "can_store", False):
                raise ValueError(f"{type(part).__name__} cannot store its output, which a norm on the output needs")
        for norm in (mixer_norm, mixer_out, ffn_norm, ffn_out):
            if norm is not None and not isinstance(norm, RMSNorm):
                raise ValueError(f"{type(norm).__name__}: this block's norms are RMS norms")
        self.width, self.mixer, self.ffn = int(width), mixer, ffn
        self.mixer_norm, self.mixer_out, self.ffn_norm, self.ffn_out = mixer_norm, mixer_out, ffn_norm, ffn_out

    @property
    def leading_norm(self) -> Norm:
        return self.mixer_norm

    def children(self) -> List[Part]:
        return [p for p in (self.mixer_norm, self.mixer, self.mixer_out, self.ffn_norm, self.ffn, self.ffn_out) if p is not None]

    def step_bytes(self, tokens: int, element_size: int) -> int:
        ffn = self.ffn.step_bytes(tokens, element_size) if self.ffn is not None else 0
        return tokens * self.width * (2 * element_size + 4) + max(self.mixer.step_bytes(tokens, element_size), ffn)

    def _read(self, ctx, norm: RMSNorm, x: torch.Tensor) -> torch.Tensor:
        left = ctx.shared.pop(self.NORMED, None)
        if left is not None and left[0] is norm and left[1] == x.data_ptr() and left[2].shape == x.shape:
            return left[2]
        h = ctx.buffer(tuple(x.shape))
        norm.forward(x, h)
        return h

    def _add(self, ctx, norm: RMSNorm, y: torch.Tensor, owed: Optional[torch.Tensor], x: torch.Tensor, following: Optional[Norm]) -> None:
        if not isinstance(following, RMSNorm):
            ops.rmsnorm_add_norm(y, norm.weight, x, norm.eps, owed)
            return
        h = ctx.buffer(tuple(x.shape))
        ops.rmsnorm_add_norm(y, norm.weight, x, norm.eps, owed, following.weight, following.eps, h)
        ctx.shared[self.NORMED] = (following, x.data_ptr(), h)

    def forward(self, ctx, x: torch.Tensor, cache) -> None:
        y = ctx.buffer(tuple(x.shape), torch.float32)
        owed = self.mixer.forward(ctx, self._read(ctx, self.mixer_norm, x), y, cache, accumulate=False)
        self._add(ctx, self.mixer_out, y, owed, x, self.ffn_norm if self.ffn is not None else ctx.next_norm)
        if self.ffn is None:
            return
        owed = self.ffn.forward(ctx, self._read(ctx, self.ffn_norm, x), y, accumulate=False)
        self._add(ctx, self.ffn_out, y, owed, x, ctx.next_norm)


class StreamBlock(Block):
    """Pre-norm with the options of a residual kept as several streams and of a token shift before the mixer:

        u = sum_s c_in[s] x_s (or x);  h = norm(u);  h <- shift(h) (mixer only);  y = sublayer(h);
        x_t <- sum_s mix[s, t] x_s + c_out[t] y   (or x += y)

    ``ffn`` None: the layer has only the mixer.  ``connections``: the two sublayers' hyper-connections (None: a
    plain residual [T, width]).  ``shift``: the token shift (None: the mixer reads the norm's output); its state,
    the last normed row of every request, is kept beside the mixer's cache (``BundleCacheSpec``).  The norms take
    ``coef=`` (:class:`carbon_engine_b200.parts.norm.GroupedRMSNorm`)."""

    def __init__(self, width: int, mixer_norm: Norm, mixer: Mixer, ffn_norm: Optional[Norm] = None,
                 ffn: Optional[FeedForward] = None, connections=None, shift=None):
        if (ffn is None) != (ffn_norm is None):
            raise ValueError("a feed-forward and its norm come together")
        if connections is not None and len(connections) != (2 if ffn is not None else 1):
            raise ValueError("one hyper-connection per sublayer")
        self.width = int(width)
        self.mixer_norm, self.mixer, self.ffn_norm, self.ffn = mixer_norm, mixer, ffn_norm, ffn
        self.connections, self.shift = connections, shift
        for part in (mixer, ffn):
            if connections is not None and part is not None and not getattr(part, "can_store", False):
                raise ValueError(f"{type(part).__name__} cannot store its output, which a residual in streams needs")

    def children(self) -> List[Part]:
        parts = [self.mixer_norm, self.mixer, self.ffn_norm, self.ffn, self.shift, *(self.connections or [])]
        return [p for p in parts if p is not None]

    def cache_spec(self):
        main = self.mixer.cache_spec()
        if self.shift is None:
            return main
        return BundleCacheSpec(main, (("shift", self.shift.state_spec()),))

    def step_bytes(self, tokens: int, element_size: int) -> int:
        h = tokens * self.width * (element_size + 4 + (4 if self.connections is not None else 0))
        ffn = self.ffn.step_bytes(tokens, element_size) if self.ffn is not None else 0
        return h + max(self.mixer.step_bytes(tokens, element_size), ffn)

    def forward(self, ctx, x: torch.Tensor, cache) -> None:
        T, W = x.shape[0], self.width
        hc = self.connections
        # the mixer
        coef = hc[0].c_in if hc is not None else None
        h = ctx.buffer((T, W))
        if self.shift is not None:
            hn = ctx.buffer((T, W), torch.float32)
            self.mixer_norm.forward(x, hn, coef=coef)
            self.shift.forward(ctx, hn, h, cache.extra["shift"])
        else:
            self.mixer_norm.forward(x, h, coef=coef)
        if hc is None:
            self.mixer.forward(ctx, h, x, cache)
        else:
            y = ctx.buffer((T, W), torch.float32)
            owed = self.mixer.forward(ctx, h, y, cache, accumulate=False)
            hc[0].write(x, y, owed)
        # the feed-forward
        if self.ffn is None:
            return
        self.ffn_norm.forward(x, h, coef=hc[1].c_in if hc is not None else None)
        if hc is None:
            self.ffn.forward(ctx, h, x)
        else:
            owed = self.ffn.forward(ctx, h, y, accumulate=False)
            hc[1].write(x, y, owed)
