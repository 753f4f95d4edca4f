"""A plain, slow implementation of the Rapovik design: whole sequences, float64, one function per mechanism.

It shares no code with the engine: it takes the configuration as the dict config.json holds and the weights
as a dict name -> tensor, runs one sequence from its first token, and keeps nothing between calls.  Keys and
values of every attention head are formed in full, recurrences go token by token, experts are looped over.

A layer normalises what each sublayer reads AND what it returns: x <- x + norm1b(mixer(norm1(x))), then
x <- x + norm2b(ff(norm2(x))).  The mixers: ``latent_attention`` (a sliding window, an interleaved rotation),
``mamba2`` (a state-space mixer with one decay per head) and ``mlstm`` (a matrix memory with exponential gates).
A span of layers may run several times in a row.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Callable, Dict, List, Optional, Tuple

import numpy as np
import torch

F = torch.float64


# ---------------------------------------------------------------------------------------------------------------
# reading a model folder
# ---------------------------------------------------------------------------------------------------------------
def read_model(folder: str) -> Tuple[dict, Dict[str, torch.Tensor]]:
    """config.json as a dict and every tensor of model.safetensors in float64 (integer tables stay integers)."""
    with open(os.path.join(folder, "config.json")) as fh:
        cfg = json.load(fh)
    with open(os.path.join(folder, "model.safetensors"), "rb") as fh:
        (n,) = struct.unpack("<Q", fh.read(8))
        header = json.loads(fh.read(n))
        data = fh.read()
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        raw, shape = data[lo:hi], tuple(meta["shape"])
        if meta["dtype"] == "BF16":
            bits = np.frombuffer(raw, dtype=np.uint16).astype(np.uint32) << 16
            t = torch.from_numpy(bits.view(np.float32).copy()).to(F)
        elif meta["dtype"] == "F32":
            t = torch.from_numpy(np.frombuffer(raw, dtype=np.float32).copy()).to(F)
        elif meta["dtype"] == "I32":
            t = torch.from_numpy(np.frombuffer(raw, dtype=np.int32).copy())
        else:
            raise ValueError(f"{name}: dtype {meta['dtype']}")
        out[name] = t.reshape(shape)
    return cfg, out


# ---------------------------------------------------------------------------------------------------------------
# norms and activations
# ---------------------------------------------------------------------------------------------------------------
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_zero_centred(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The layers' and the model's norm: the stored weight is the deviation from 1."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    return -softplus(-z)


def soft_cap(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


def clamped_glu(gate: torch.Tensor, up: torch.Tensor, limit: float) -> torch.Tensor:
    """g = min(gate, limit), u = up cut to [-limit, limit]; g sigmoid(1.702 g) (u + 1)."""
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


# ---------------------------------------------------------------------------------------------------------------
# latent attention
# ---------------------------------------------------------------------------------------------------------------
def rotate_neighbours(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, size]: of the first ``dims`` elements, 2i turns with 2i + 1 by position * base^(-2i/dims)."""
    out = x.clone()
    for i in range(dims // 2):
        ang = positions.to(F) * base ** (-2.0 * i / dims)
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def window_softmax(scores: torch.Tensor, window: int) -> torch.Tensor:
    """Row i of a [T, T] score table sees the columns j with 0 <= i - j < window (window 0: all j <= i)."""
    out = torch.zeros_like(scores)
    for i in range(scores.shape[0]):
        lo = max(0, i - window + 1) if window else 0
        row = scores[i, lo:i + 1]
        e = torch.exp(row - row.max())
        out[i, lo:i + 1] = e / e.sum()
    return out


def latent_attention(w: Dict[str, torch.Tensor], p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, dr, dv, r = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    pos, dims, base = torch.arange(T), int(m["rot"]["dims"]), float(m["rot"]["base"])
    z = h @ w[f"{p}.dkv"].T
    c = unit_rms(z[:, :r], eps) * w[f"{p}.dkv.norm"]
    k_rot = rotate_neighbours(z[:, None, r:], pos, dims, base)[:, 0]
    q = (h @ w[f"{p}.q"].T).view(T, H, d + dr)
    q_rot = rotate_neighbours(q[..., d:], pos, dims, base)
    k = (c @ w[f"{p}.uk"].T).view(T, H, d)
    v = (c @ w[f"{p}.uv"].T).view(T, H, dv)
    window = int((m.get("mask") or {}).get("size", 0))
    heads = []
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].T + q_rot[:, i] @ k_rot.T) * float(m["scale"])
        heads.append(window_softmax(s, window) @ v[:, i])
    return torch.cat(heads, dim=-1) @ w[f"{p}.o"].T


# ---------------------------------------------------------------------------------------------------------------
# the state-space mixer
# ---------------------------------------------------------------------------------------------------------------
def causal_conv(x: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, K] (the last column weighs the current token, zeros before the start), bias [C]."""
    T, C = x.shape
    K = taps.shape[1]
    padded = torch.cat([torch.zeros((K - 1, C), dtype=F), x], dim=0)
    y = bias[None, :].expand(T, C).clone()
    for j in range(K):
        y = y + padded[j:j + T] * taps[:, j][None, :]
    return y


def state_space_walk(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, a: float, skip: float) -> torch.Tensor:
    """One head: x [T, dv], B, C [T, N], dt [T] -> y [T, dv].  S <- exp(-a dt) S + dt B x^T; y = S^T C + skip x."""
    T = x.shape[0]
    S = torch.zeros((B.shape[1], x.shape[1]), dtype=F)
    out = torch.zeros_like(x)
    for t in range(T):
        S = torch.exp(-a * dt[t]) * S + dt[t] * torch.outer(B[t], x[t])
        out[t] = S.T @ C[t] + skip * x[t]
    return out


def mamba2(w: Dict[str, torch.Tensor], p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, dv, N, G, parts = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m["norm_groups"])
    inner = H * dv
    zxbcdt = h @ w[f"{p}.in"].T
    z, xbc, dt = zxbcdt[:, :inner], zxbcdt[:, inner:2 * inner + 2 * G * N], zxbcdt[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[f"{p}.conv"], w[f"{p}.conv.b"]))
    x = xbc[:, :inner].reshape(T, H, dv)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + w[f"{p}.dt_bias"][None, :])
    y = torch.zeros((T, H, dv), dtype=F)
    for i in range(H):
        g = i // (H // G)
        y[:, i] = state_space_walk(x[:, i], B[:, g], C[:, g], dt[:, i], math.exp(float(w[f"{p}.A_log"][i])), float(w[f"{p}.D"][i]))
    y = y.reshape(T, inner) * silu(z)
    y = unit_rms(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * w[f"{p}.norm"]
    return y @ w[f"{p}.o"].T


# ---------------------------------------------------------------------------------------------------------------
# the matrix memory
# ---------------------------------------------------------------------------------------------------------------
def matrix_memory_walk(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, log_i: torch.Tensor, log_f: torch.Tensor) -> torch.Tensor:
    """One head: q, k [T, d], v [T, dv], log_i, log_f [T] -> o [T, dv].  The running maximum m starts at 0."""
    T, d = q.shape
    S, n, m = torch.zeros((d, v.shape[1]), dtype=F), torch.zeros(d, dtype=F), 0.0
    out = torch.zeros((T, v.shape[1]), dtype=F)
    for t in range(T):
        i, f = float(log_i[t]), float(log_f[t])
        new = max(f + m, i)
        keep, write = math.exp(f + m - new), math.exp(i - new)
        S = keep * S + write * torch.outer(k[t], v[t])
        n = keep * n + write * k[t]
        m = new
        out[t] = (S.T @ q[t]) / (max(abs(float(n @ q[t])), math.exp(-m)) + 1e-6)
    return out


def mlstm(w: Dict[str, torch.Tensor], p: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv, cap = int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"])
    q = (h @ w[f"{p}.q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[f"{p}.k"].T).reshape(T, H, d)
    v = (h @ w[f"{p}.v"].T).reshape(T, H, dv)
    log_i = soft_cap(h @ w[f"{p}.i"].T + w[f"{p}.i.b"][None, :], cap)
    log_f = log_sigmoid(soft_cap(h @ w[f"{p}.f"].T + w[f"{p}.f.b"][None, :], cap))
    o = torch.stack([matrix_memory_walk(q[:, j], k[:, j], v[:, j], log_i[:, j], log_f[:, j]) for j in range(H)], dim=1)
    o = unit_rms(o, eps).reshape(T, H * dv) * w[f"{p}.norm"] * torch.sigmoid(h @ w[f"{p}.g"].T)
    return o @ w[f"{p}.o"].T


# ---------------------------------------------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------------------------------------------
def gated_ff(w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, limit: float, biases: bool) -> torch.Tensor:
    b = lambda name: w[f"{p}.{name}.b"][None, :] if biases else 0.0
    return clamped_glu(h @ w[f"{p}.gate"].T + b("gate"), h @ w[f"{p}.up"].T + b("up"), limit) @ w[f"{p}.down"].T + b("down")


def route(z: torch.Tensor, correction: torch.Tensor, router: dict, margin: Optional[list] = None) -> Tuple[List[int], List[float]]:
    """One token's router logits -> the chosen experts (best first) and their weights.  ``margin`` receives how clear the
    choice was: the smallest gap, in scores, between the last kept group and the first dropped one and between the last
    chosen expert and the first one passed over."""
    E, top = int(router["experts"]), int(router["top"])
    s = torch.sigmoid(z)
    choice = s + correction
    allowed = list(range(E))
    gap = math.inf
    groups = router.get("groups")
    if groups:
        n, keep = int(groups["count"]), int(groups["keep"])
        size = E // n
        score = [sum(sorted((float(choice[g * size + j]) for j in range(size)), reverse=True)[:2]) for g in range(n)]
        order = sorted(range(n), key=lambda g: -score[g])
        allowed = [e for e in range(E) if e // size in order[:keep]]
        if keep < n:
            gap = score[order[keep - 1]] - score[order[keep]]
    ranked = sorted(allowed, key=lambda e: -float(choice[e]))
    if top < len(ranked):
        gap = min(gap, float(choice[ranked[top - 1]] - choice[ranked[top]]))
    if margin is not None:
        margin.append(gap)
    return ranked[:top], [float(s[e]) for e in ranked[:top]]


def moe_ff(w: Dict[str, torch.Tensor], p: str, mlp: dict, h: torch.Tensor, margins: Optional[list] = None) -> torch.Tensor:
    """``margins`` receives one number per token: the gap of :func:`route`."""
    out = torch.zeros_like(h)
    z = h @ w[f"{p}.router"].T
    for t in range(h.shape[0]):
        chosen, weights = route(z[t], w[f"{p}.correction"], mlp["router"], margins)
        for e, g in zip(chosen, weights):
            out[t] += g * gated_ff(w, f"{p}.e{e}", h[t:t + 1], float(mlp["expert"]["limit"]), False)[0]
    if mlp.get("shared"):
        out = out + gated_ff(w, f"{p}.shared", h, float(mlp["shared"]["limit"]), False)
    return out


# ---------------------------------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------------------------------
MIXERS = {"latent_attention": latent_attention, "mamba2": mamba2, "mlstm": mlstm}


def layer_runs(cfg: dict) -> List[int]:
    order = list(range(len(cfg["layers"])))
    loop = cfg.get("loop")
    if not loop:
        return order
    a, b = int(loop["start"]), int(loop["stop"])
    return order[:a] + order[a:b] * int(loop["times"]) + order[b:]


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], tap: Optional[Callable] = None,
            margins: Optional[list] = None, round_input: Optional[Callable] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence from its first token.  ``tap(i, x)`` sees the residual after the i-th layer run;
    ``margins`` receives, per run of a mixture layer, a list with every token's router margin; ``round_input`` is applied
    to what the sublayers read (to see what a rounding of the activations does)."""
    eps = float(cfg["norm"]["eps"])
    rd = round_input or (lambda t: t)
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)].to(F)
    for run, i in enumerate(layer_runs(cfg)):
        p, layer = f"l{i}", cfg["layers"][i]
        y = MIXERS[layer["type"]](w, f"{p}.mix", layer["mixer"], rd(norm_zero_centred(x, w[f"{p}.norm1"], eps)), eps)
        x = x + norm_zero_centred(y, w[f"{p}.norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rd(norm_zero_centred(x, w[f"{p}.norm2"], eps))
            if mlp["kind"] == "dense":
                y = gated_ff(w, f"{p}.mlp", h, float(mlp["limit"]), True)
            else:
                per_token: list = []
                y = moe_ff(w, f"{p}.mlp", mlp, h, per_token)
                if margins is not None:
                    margins.append(per_token)
            x = x + norm_zero_centred(y, w[f"{p}.norm2b"], eps)
        if tap is not None:
            tap(run, x)
    return norm_zero_centred(x, w["final.norm"], eps) @ w["head"].T
