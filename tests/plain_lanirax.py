"""A plain, slow implementation of the Lanirax design: whole sequences, float64, one function per mechanism.

It shares no code with the engine: it takes the configuration as the dict config.json holds and the weights
as a dict name -> tensor, runs one sequence from its first token, and keeps nothing between calls.

A layer has no norm in front of a sublayer; the norm is taken of the weighted residual plus the sublayer's output:
x <- norm1(alpha x + mixer(x)), then x <- norm2(alpha x + ff(x)).  The mixers: ``attention`` (no rotation: a temperature
that grows with the query's position and a penalty that grows with the distance of the key) and ``parallel`` (windowed
softmax attention whose values are the projected keys, with a stretched rotation, a norm behind the rotation and a sink per
head, beside the gated delta rule with one decay per head; half the sum of the two outputs, each normed over the width).
The feed-forward is a mixture of gated experts.  A layer may run another layer's weights.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional, Tuple

import torch

F = torch.float64
Weights = Dict[str, torch.Tensor]


# ---------------------------------------------------------------------------------------------------------------
# reading a model folder
# ---------------------------------------------------------------------------------------------------------------
def read_model(folder: str) -> Tuple[dict, Weights]:
    """config.json as a dict and every tensor of model.safetensors, floats in float64."""
    with open(os.path.join(folder, "config.json")) as fh:
        cfg = json.load(fh)
    with open(os.path.join(folder, "model.safetensors"), "rb") as fh:
        (n,) = struct.unpack("<Q", fh.read(8))
        header = json.loads(fh.read(n))
        data = bytearray(fh.read())
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        dt = {"F32": torch.float32, "BF16": torch.bfloat16, "I32": torch.int32}[meta["dtype"]]
        t = torch.frombuffer(data[lo:hi], dtype=dt).reshape(meta["shape"])
        out[name] = t.to(F) if t.is_floating_point() else t.clone()
    return cfg, out


# ---------------------------------------------------------------------------------------------------------------
# norms and activations
# ---------------------------------------------------------------------------------------------------------------
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * weight


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


# ---------------------------------------------------------------------------------------------------------------
# positions
# ---------------------------------------------------------------------------------------------------------------
def stretched_frequencies(dims: int, base: float, scaling: Optional[dict]) -> Tuple[List[float], float]:
    """(one frequency per pair, the factor on cosine and sine): fast pairs keep base^(-2i/dims), slow ones are divided by
    ``factor``, with a linear ramp between the pairs that turn ``fast`` and ``slow`` times within ``original`` positions."""
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return freqs, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(index_of(float(scaling["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(1.0, max(0.0, (i - lo) / max(hi - lo, 0.001)))
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_neighbours(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, size], row t at position t: of the first ``dims`` elements, 2i turns with 2i + 1."""
    T, dims = x.shape[0], int(rot["dims"])
    freqs, amp = stretched_frequencies(dims, float(rot["base"]), rot.get("scaling"))
    out = x.clone()
    for i, f in enumerate(freqs):
        ang = torch.arange(T, dtype=F) * f
        c, s = (amp * torch.cos(ang))[:, None], (amp * torch.sin(ang))[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def query_temperature(T: int, coef: float, every: float) -> torch.Tensor:
    """One factor per position p: 1 + coef ln(floor((p + 1) / every) + 1)."""
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0) for p in range(T)], dtype=F)


def distance_slopes(heads: int) -> List[float]:
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


# ---------------------------------------------------------------------------------------------------------------
# softmax attention
# ---------------------------------------------------------------------------------------------------------------
def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: int = 0,
                      sink: Optional[torch.Tensor] = None, slopes: Optional[List[float]] = None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query i sees the keys j with 0 <= i - j (< window); slope_h (i - j) comes off
    the score; exp(sink_h) joins the denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    dist = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    hidden = dist < 0
    if window > 0:
        hidden = hidden | (dist >= window)
    out = torch.zeros((T, H, v.shape[2]), dtype=F)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if slopes is not None:
            s = s - slopes[h] * dist.to(F)
        s = s.masked_fill(hidden, float("-inf"))
        top = s.max(dim=-1, keepdim=True).values
        if sink is not None:
            top = torch.clamp(top, min=float(sink[h]))
        e = torch.exp(s - top)
        total = e.sum(-1, keepdim=True)
        if sink is not None:
            total = total + torch.exp(sink[h] - top)
        out[:, h] = (e @ v[:, g]) / total
    return out


def distance_attention(w: Weights, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    """The mixer ``attention``."""
    T, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms_norm((h @ w[f"{p}.q"].T).reshape(T, H, d), w[f"{p}.q.norm"], eps)
    k = rms_norm((h @ w[f"{p}.k"].T).reshape(T, G, d), w[f"{p}.k.norm"], eps)
    v = (h @ w[f"{p}.v"].T).reshape(T, G, dv)
    if m.get("q_temp"):
        q = q * query_temperature(T, float(m["q_temp"]["coef"]), float(m["q_temp"]["every"]))[:, None, None]
    out = softmax_attention(q, k, v, float(m["scale"]), slopes=distance_slopes(H))
    return out.reshape(T, H * dv) @ w[f"{p}.o"].T


def tied_window_attention(w: Weights, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    """The left member of ``parallel``: the values are the keys as projected."""
    T, H, G, d = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = (h @ w[f"{p}.q"].T).reshape(T, H, d)
    v = (h @ w[f"{p}.k"].T).reshape(T, G, d)
    turn = lambda x: rotate_neighbours(x, m["rot"]) if m.get("rot") else x
    q, k = unit_rms(turn(q), eps), unit_rms(turn(v), eps)
    window = int(m["mask"]["size"]) if m.get("mask") else 0
    out = softmax_attention(q, k, v, float(m["scale"]), window=window, sink=w[f"{p}.sink"])
    return out.reshape(T, H * d) @ w[f"{p}.o"].T


# ---------------------------------------------------------------------------------------------------------------
# the gated delta rule
# ---------------------------------------------------------------------------------------------------------------
def short_convolution(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, K]: y_t = sum_j taps[:, K - 1 - j] x_(t - j), zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for j in range(min(K, T)):
        y[j:] += x[:T - j] * taps[:, K - 1 - j]
    return y


def unit_length(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_walk(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor) -> torch.Tensor:
    """One head: q, k [T, d], v [T, dv], g and beta [T] -> o [T, dv]."""
    S = torch.zeros((q.shape[1], v.shape[1]), dtype=F)
    rows = []
    for t in range(q.shape[0]):
        S = g[t] * S
        u = beta[t] * (v[t] - k[t] @ S)
        S = S + k[t][:, None] * u[None, :]
        rows.append(q[t] @ S)
    return torch.stack(rows)


def gated_delta(w: Weights, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    """The right member of ``parallel``."""
    T, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    path = lambda name: silu(short_convolution(h @ w[f"{p}.{name}"].T, w[f"{p}.{name}.conv"]))
    q = unit_length(path("q").reshape(T, G, d)) / math.sqrt(d)
    k = unit_length(path("k").reshape(T, G, d))
    v = path("v").reshape(T, H, dv)
    beta = torch.sigmoid(h @ w[f"{p}.b"].T)
    g = torch.exp(-torch.exp(w[f"{p}.A_log"]) * softplus(h @ w[f"{p}.a"].T + w[f"{p}.dt_bias"]))
    o = torch.stack([delta_walk(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], g[:, i], beta[:, i]) for i in range(H)], dim=1)
    o = rms_norm(o, w[f"{p}.norm"], eps) * silu(h @ w[f"{p}.g"].T).reshape(T, H, dv)
    return o.reshape(T, H * dv) @ w[f"{p}.o"].T


def parallel(w: Weights, p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    left = rms_norm(tied_window_attention(w, f"{p}.left", m["left"], h, eps), w[f"{p}.left.out"], eps)
    right = rms_norm(gated_delta(w, f"{p}.right", m["right"], h, eps), w[f"{p}.right.out"], eps)
    return 0.5 * (left + right)


# ---------------------------------------------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------------------------------------------
def expert(w: Weights, p: str, h: torch.Tensor) -> torch.Tensor:
    return (silu(h @ w[f"{p}.gate"].T) * (h @ w[f"{p}.up"].T)) @ w[f"{p}.down"].T


def mixture(w: Weights, p: str, mlp: dict, h: torch.Tensor, margins: Optional[list] = None) -> torch.Tensor:
    """``margins`` receives, per token, the gap between the last logit chosen and the first one not."""
    top = int(mlp["router"]["top"])
    z = h @ w[f"{p}.router"].T + w[f"{p}.router.b"]
    out = torch.zeros_like(h)
    if margins is not None:
        ranked = torch.sort(z, dim=-1, descending=True).values
        margins.append((ranked[:, top - 1] - ranked[:, top]).tolist() if top < z.shape[1] else [float("inf")] * h.shape[0])
    for t in range(h.shape[0]):
        chosen = torch.sort(z[t], descending=True, stable=True).indices[:top]
        weight = torch.exp(z[t][chosen] - z[t][chosen].max())
        weight = weight / weight.sum()
        for e, c in zip(chosen.tolist(), weight):
            out[t] += c * expert(w, f"{p}.e{e}", h[t])
    return out


# ---------------------------------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------------------------------
MIXERS = {"attention": distance_attention, "parallel": parallel}


def owner(layers: list, i: int) -> int:
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def forward(cfg: dict, weights: Weights, tokens: List[int], layers_out: Optional[list] = None, rounding=None,
            margins: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` receives the residual after every layer, ``margins`` the routers' (see
    :func:`mixture`).  ``rounding``: a function applied to what every sublayer reads (to see how far rounding alone moves the
    result)."""
    w = {k: v.to(F) if v.is_floating_point() else v for k, v in weights.items()}
    read = rounding if rounding is not None else lambda x: x
    eps, alpha = float(cfg["norm"]["eps"]), float(cfg["postln_alpha"])
    x = rms_norm(w["embed"][torch.tensor(tokens, dtype=torch.long)], w["embed.norm"], eps)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{owner(cfg['layers'], i)}"
        x = rms_norm(alpha * x + MIXERS[layer["type"]](w, f"{p}.mix", layer["mixer"], read(x), eps), w[f"{p}.norm1"], eps)
        if layer.get("mlp") is not None:
            x = rms_norm(alpha * x + mixture(w, f"{p}.mlp", layer["mlp"], read(x), margins), w[f"{p}.norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return read(rms_norm(x, w["final.norm"], eps)) @ w["head"].T
