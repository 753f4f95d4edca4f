"""Small Lanirax configurations for the tests.

They differ from one another in every size and option: widths and vocabularies that are no powers of two; which mixer comes first;
head counts and groups (one key head for all, one per query head, groups of two and three), value heads smaller and larger than the
keys, the rotated part (a part of the head, all of it, none), stretched rotations whose ramp lies inside, at the start and beyond the
rotated pairs and a plain one, windows of one token up to more than any test sequence, 1 to 6 taps, key heads of the delta rule fewer
than and as many as its heads, temperatures that step often, once and never, weights of the residual below, at and above 1; no
feed-forward, mixtures of which one, some and all experts are chosen; layers that run an earlier and a later layer's weights.
"""
from __future__ import annotations

from typing import Dict, Optional

from munizen_cases import Harness, rel_err  # noqa: F401  (the harness steps any architecture's folder)


def moe(experts=6, top=2, ff=12):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def stretched(factor=3.0, original=64, fast=8.0, slow=0.7):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attention(heads=4, kv_heads=2, dim=12, vdim=20, scale=0.4, temp=(0.3, 7), mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def pair(heads=4, kv_heads=2, dim=16, scale=0.5, window=9, rot_dims=8, base=300.0, scaling: Optional[dict] = "default", r_heads=4, r_kv=2,
         r_dim=10, r_vdim=14, conv=4, mlp=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if window:
        left["mask"] = {"size": window}
    if rot_dims:
        left["rot"] = {"dims": rot_dims, "base": base}
        if scaling is not None:
            left["rot"]["scaling"] = stretched() if scaling == "default" else scaling
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": left, "right": {"heads": r_heads, "kv_heads": r_kv, "dim": r_dim, "vdim": r_vdim, "conv": conv}}}


def shared(layer: dict, of: int) -> dict:
    return dict(layer, weights_of=of)


def config(layers, width=40, vocab=97, eps=1e-5, alpha=1.3, max_positions=1024):
    return {"architecture": "Lanirax", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "postln_alpha": alpha,
            "max_position_embeddings": max_positions}


_a0, _a1 = pair(mlp=moe()), attention(mlp=moe(experts=9, top=4, ff=10))
_b1 = attention(heads=3, kv_heads=3, dim=10, vdim=6, scale=0.7, temp=None, mlp=moe(experts=5, top=1, ff=17))
_t0 = pair(heads=4, kv_heads=2, dim=64, scale=0.2, window=50, rot_dims=32, r_heads=2, r_kv=1, r_dim=32, r_vdim=32, conv=3,
           mlp=moe(experts=8, top=3, ff=32))
CASES: Dict[str, dict] = {
    # both mixers; the pair again with the first layer's weights; a last layer without a feed-forward
    "A": config([_a0, _a1, shared(_a0, 0), pair(heads=2, kv_heads=2, dim=8, window=21, rot_dims=8, scaling=stretched(1.0, 20, 2.0, 0.1),
                                                r_heads=3, r_kv=3, r_dim=7, r_vdim=5, conv=1)]),
    # attention first, running the weights of a LATER layer; every expert chosen; no rotation; a window of one token; alpha below 1
    "B": config([shared(_b1, 2), pair(heads=6, kv_heads=1, dim=9, scale=1.1, window=1, rot_dims=0, r_heads=1, r_kv=1, r_dim=20, r_vdim=6, conv=6,
                                      mlp=moe(experts=4, top=4, ff=9)), _b1, attention(heads=2, kv_heads=1, dim=7, vdim=11, temp=(1.5, 500))],
                width=36, vocab=61, eps=1e-3, alpha=0.6),
    # a window longer than every sequence, a plain rotation, a ramp that starts past the rotated pairs; a chain of shared layers
    "C": config([pair(heads=3, kv_heads=1, dim=12, window=4096, rot_dims=4, scaling=None, r_heads=6, r_kv=2, r_dim=4, r_vdim=9, conv=2, mlp=moe(7, 3, 8)),
                 attention(heads=6, kv_heads=2, dim=5, vdim=5, temp=(0.2, 1), mlp=None),
                 shared(attention(heads=6, kv_heads=2, dim=5, vdim=5, temp=(0.2, 1), mlp=None), 1),
                 pair(heads=2, kv_heads=1, dim=10, window=30, rot_dims=10, base=5000.0, scaling=stretched(40.0, 100000, 0.001, 0.0005), r_heads=2,
                      r_kv=1, r_dim=12, r_vdim=8, conv=5, mlp=moe(3, 2, 21))], width=44, vocab=75, alpha=2.5),
    # sizes of the tensor-core kernels: heads of 64 (tcgen05 flash, TMA decode) and of 32 (mma.sync flash, cp.async decode)
    "T": config([_t0, attention(heads=4, kv_heads=1, dim=32, vdim=32, scale=0.3, temp=(0.3, 20), mlp=moe(experts=16, top=4, ff=24)),
                 attention(heads=2, kv_heads=2, dim=64, vdim=64, scale=0.2, temp=(0.2, 33), mlp=None), shared(_t0, 0)], width=64, vocab=151),
    # the same with values of another size than the keys (the masked-attention family's tensor-core kernel), wider
    "V": config([attention(heads=8, kv_heads=2, dim=32, vdim=48, scale=0.25, mlp=moe(experts=16, top=2, ff=48)),
                 pair(heads=2, kv_heads=1, dim=32, scale=0.3, window=40, rot_dims=16, r_heads=2, r_kv=2, r_dim=64, r_vdim=128, conv=4,
                      mlp=moe(experts=12, top=3, ff=40)),
                 attention(heads=4, kv_heads=4, dim=64, vdim=16, scale=0.2, temp=(0.5, 11), mlp=None)], width=256, vocab=300, alpha=1.0),
}
#: one layer alone, for looking at a mechanism by itself
SINGLE = {
    "attention": config([attention()]),
    "attention_plain_temperature": config([attention(temp=None, heads=3, kv_heads=1)]),
    "pair": config([pair()]),
    "pair_one_token_window": config([pair(window=1, rot_dims=16)]),
    "pair_no_window_no_stretch_one_tap": config([pair(window=0, scaling=None, conv=1)]),
    "pair_wide_state_keys": config([pair(r_heads=1, r_kv=1, r_dim=136, r_vdim=6, dim=24, rot_dims=6)]),
    "experts": config([attention(heads=1, kv_heads=1, dim=4, vdim=4, mlp=moe())]),
    "experts_one_chosen": config([attention(heads=1, kv_heads=1, dim=4, vdim=4, mlp=moe(experts=11, top=1))]),
    "experts_all_chosen": config([attention(heads=1, kv_heads=1, dim=4, vdim=4, mlp=moe(experts=3, top=3))]),
    "shared": config([pair(mlp=moe()), shared(pair(mlp=moe()), 0)]),
}


def write_model(raw: dict, folder: str, seed: int = 3, change=None) -> str:
    """A random model folder; ``change(tensors)`` may edit the stored tensors (so that what random weights would hide shows)."""
    import os

    import carbon_engine_b200.models  # noqa: F401
    from carbon_engine_b200.config.lanirax import LaniraxConfig
    from carbon_engine_b200.weights.loader import write_random_model
    out = write_random_model(LaniraxConfig.from_dict(dict(raw)), folder, seed=seed)
    path = os.path.join(out, "model.safetensors")
    from helpers import read_raw_safetensors, write_safetensors_plain
    t = read_raw_safetensors(path)
    for name in t:
        # matrices of 0.02 would leave the sublayers' outputs, which are added to a residual of unit size, without weight
        if t[name].dim() == 2 and not name.endswith(".conv") and name != "embed":
            gain = 2.0 if name.endswith("router") else 1.0
            t[name] = (t[name].float() * (gain * 50.0 * t[name].shape[1] ** -0.5)).to(t[name].dtype)
    if change is not None:
        change(t)
    write_safetensors_plain(path, t)
    return out
