"""One-layer Lanirax models in which every query scores the marker token's key far above hundreds of others.

The first embedding element is the same large number for every token, so the first element of the normed embedding is nearly
constant; one query element reads it, and the same key element reads the direction of the marker's embedding: behind the norm per
head (which another, constant key element keeps alike for all tokens) it is large for the marker and noise for all others.  The
second embedding element is 1 for every token and -1 for the marker; one value element reads it and the output product spreads it
over the width: the output turns round where the marker is seen, which a norm of the output does not hide.
"""
from __future__ import annotations

import torch

from lanirax_cases import attention, config, pair, write_model

MARKER, ORDINARY = 7, 9
WIDTH = 48


def _matrices(t: dict, prefix: str, heads: int, kv_heads: int, d: int, dv: int, tied: bool) -> None:
    # element j of a head carries the score, element j + 1 holds the keys' norm in place; they lie past every rotated part used here
    j = d - 6
    jv = j + 2 if tied else dv - 3
    mark = t["embed"][MARKER].float().clone()
    mark[:2] = 0.0
    mark = mark / mark.norm()
    first, second = torch.zeros(WIDTH), torch.zeros(WIDTH)
    first[0], second[1] = 1.0, 1.0
    # even and odd heads write different patterns, so that a head's share shows behind a norm too
    signs = [torch.tensor([1.0 if (3 * c) % 7 < 4 else -1.0 for c in range(WIDTH)]),
             torch.tensor([1.0 if (5 * c) % 11 < 6 else -1.0 for c in range(WIDTH)])]
    bf = torch.bfloat16
    for n in ("q", "k", "v", "o"):
        if f"{prefix}.{n}" in t:
            t[f"{prefix}.{n}"] = (t[f"{prefix}.{n}"].float() * 0.1).to(bf)
    for h in range(heads):
        t[f"{prefix}.q"][h * d + j] = (4.0 * first).to(bf)
        t[f"{prefix}.o"][:, h * dv + jv] = (0.6 * signs[h % 2]).to(bf)
    for h in range(kv_heads):
        t[f"{prefix}.k"][h * d + j] = (0.8 * mark).to(bf)
        t[f"{prefix}.k"][h * d + j + 1] = (2.0 * first).to(bf)
        t[f"{prefix}.k" if tied else f"{prefix}.v"][h * dv + jv] = (2.0 * second).to(bf)


def _embedding(t: dict) -> None:
    e = t["embed"].float() * 50.0
    e[:, 0], e[:, 1] = 3.0, 1.0
    e[MARKER, 1] = -1.0
    t["embed"], t["embed.norm"] = e.to(torch.bfloat16), torch.ones(WIDTH)


def distance_model(folder: str, d: int = 16, dv: int = 16, heads: int = 4, kv_heads: int = 2, strength: float = 40.0) -> str:
    """An attention layer: the penalty on distance (steep in the first heads, slight in the last) is set against the marker's score."""
    def change(t):
        _embedding(t)
        _matrices(t, "l0.mix", heads, kv_heads, d, dv, tied=False)
        t["l0.mix.q.norm"], t["l0.mix.k.norm"] = torch.ones(d), torch.ones(d)
    return write_model(config([attention(heads, kv_heads, d, dv, scale=strength / d, temp=(0.2, 50))], width=WIDTH, vocab=50, alpha=1.0),
                       folder, seed=21, change=change)


def window_model(folder: str, window: int, d: int = 16, heads: int = 4, kv_heads: int = 2, sink=None, strength: float = 40.0) -> str:
    """A pair layer in which only the attention counts (the delta rule's output norm has weight zero)."""
    def change(t):
        _embedding(t)
        _matrices(t, "l0.mix.left", heads, kv_heads, d, d, tied=True)
        t["l0.mix.right.out"] = torch.zeros(WIDTH)
        t["l0.mix.left.sink"] = torch.full((heads,), -30.0) if sink is None else torch.tensor(sink, dtype=torch.float32)
    raw = config([pair(heads=heads, kv_heads=kv_heads, dim=d, window=window, rot_dims=8, scale=strength / d, r_heads=1, r_kv=1, r_dim=4,
                       r_vdim=4, conv=2)], width=WIDTH, vocab=50, alpha=1.0)
    return write_model(raw, folder, seed=21, change=change)
