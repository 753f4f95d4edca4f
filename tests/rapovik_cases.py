"""Small Rapovik configurations for the tests.

They differ from one another in every size and option: widths and vocabularies that are no powers of two; the order of the three
mixers and which comes first; state sizes against value sizes, one group and several, 1 to 5 taps, norm parts that are fewer than,
as many as and more than the groups or cut through heads; matrix memories with wider keys than values and the reverse, small caps;
latent attention with and without a window, the rotated part turned whole or in part, latents smaller and larger than a head; no
feed-forward, dense ones and mixtures in any order; mixtures without groups, with groups of one expert, with every group kept,
with every expert chosen, with and without a shared expert, limits that differ between the experts and the shared one; spans of
layers that run once, twice and three times, at the start, in the middle and all.
"""
from __future__ import annotations

from typing import Dict

from munizen_cases import Harness, rel_err  # noqa: F401  (the harness steps any architecture's folder)


def dense(ff=40, limit=1.1):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts=6, top=2, ff=12, groups=(3, 2), shared=20, limit=0.9, shared_limit=0.6):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def attention(heads=3, dim=12, rot_dim=8, vdim=20, kv_rank=14, scale=0.25, rot_dims=None, base=500.0, window=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"dims": rot_dims or rot_dim, "base": base}}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def mamba(heads=4, vdim=10, state=12, groups=2, conv=4, norm_groups=2, mlp=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}, "mlp": mlp}


def mlstm(heads=3, dim=8, vdim=12, gate_cap=15.0, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}, "mlp": mlp}


def config(layers, width=40, vocab=97, eps=1e-5, loop=None, max_positions=1024):
    raw = {"architecture": "Rapovik", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
           "max_position_embeddings": max_positions}
    if loop:
        raw["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return raw


CASES: Dict[str, dict] = {
    # all three mixers, a span in the middle run twice, a window, mixtures with groups
    "A": config([mamba(mlp=dense()), mlstm(mlp=moe()), attention(window=21, mlp=moe(experts=8, top=3, groups=(2, 1), ff=10)),
                 mamba(heads=2, vdim=6, state=20, groups=1, conv=3, norm_groups=1, mlp=dense(24, 0.4))], loop=(1, 3, 2)),
    # attention first, without a window, a part of the rotated part turned; no feed-forward; one tap; parts that cut through heads;
    # groups of one expert; no shared expert; the first layers run three times
    "B": config([attention(heads=1, dim=10, rot_dim=6, vdim=7, kv_rank=30, rot_dims=4, base=77.0, mlp=None),
                 mlstm(heads=2, dim=20, vdim=6, gate_cap=1.5, mlp=moe(experts=5, top=3, groups=(5, 4), shared=8, limit=3.0, shared_limit=0.3)),
                 mamba(heads=3, vdim=8, state=5, groups=3, conv=1, norm_groups=4, mlp=moe(experts=7, top=7, groups=None, ff=9, shared=None)),
                 mlstm(heads=1, dim=5, vdim=17, mlp=None)], width=36, vocab=61, eps=1e-6, loop=(0, 2, 3)),
    # matrix memory first; a narrow window; five taps; all groups kept; the whole model twice
    "C": config([mlstm(heads=4, dim=4, vdim=4, gate_cap=6.0, mlp=dense(33, 2.0)),
                 mamba(heads=6, vdim=4, state=9, groups=3, conv=5, norm_groups=1, mlp=None),
                 attention(heads=5, dim=4, rot_dim=2, vdim=9, kv_rank=9, scale=0.6, base=1e4, window=5, mlp=moe(experts=8, top=4, groups=(2, 2), ff=7, shared=5))],
                width=44, vocab=75, loop=(0, 3, 2)),
    # sizes of the tensor-core kernels (multiples of 16), eight heads so that single tokens pack them into one tile; no loop
    "T": config([attention(heads=8, dim=16, rot_dim=16, vdim=32, kv_rank=48, scale=0.18, base=1e4, window=50, mlp=dense(96, 1.5)),
                 mamba(heads=4, vdim=32, state=32, groups=2, conv=4, norm_groups=4, mlp=moe(experts=8, top=2, ff=32, groups=(4, 2), shared=48)),
                 mlstm(heads=2, dim=32, vdim=64, mlp=moe(experts=8, top=3, ff=24, groups=(4, 2), shared=64))], width=64, vocab=151),
    # wider: a latent row of 192 + 32, state heads of more than 64 and of more than 128 key channels
    "V": config([mamba(heads=2, vdim=64, state=136, groups=1, conv=2, norm_groups=2, mlp=moe(experts=16, top=4, ff=48, groups=(4, 2), shared=96)),
                 attention(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=192, scale=0.1, base=1e4, window=64, mlp=dense(272, 1.0)),
                 mlstm(heads=2, dim=96, vdim=128, gate_cap=4.0, mlp=dense(128, 0.8))], width=192, vocab=300, loop=(1, 2, 2)),
}
#: one layer alone, for looking at a mechanism by itself
_tiny = dict(heads=1, dim=4, vdim=4)
SINGLE = {
    "attention": config([attention()]),
    "attention_window": config([attention(window=7, rot_dims=2)]),
    "attention_window_of_one": config([attention(window=1)]),
    "mamba": config([mamba()]),
    "mamba_one_tap_one_group": config([mamba(heads=2, vdim=9, state=7, groups=1, conv=1, norm_groups=3)], width=34),
    "mamba_wide_state": config([mamba(heads=1, vdim=8, state=136, groups=1, conv=3, norm_groups=1)]),
    "mlstm": config([mlstm()]),
    "mlstm_small_cap_odd_sizes": config([mlstm(heads=2, dim=9, vdim=5, gate_cap=0.7)], width=34),
    "mlstm_wide_keys": config([mlstm(heads=1, dim=136, vdim=6)]),
    "dense": config([mlstm(**_tiny, mlp=dense(33, 0.5))]),
    "experts": config([mlstm(**_tiny, mlp=moe())]),
    "experts_all_chosen_no_shared": config([mlstm(**_tiny, mlp=moe(experts=7, top=7, groups=None, shared=None))]),
    "looped": config([mamba(mlp=None)], loop=(0, 1, 3)),
}


def write_model(raw: dict, folder: str, seed: int = 3, change=None) -> str:
    """A random model folder; ``change(tensors)`` may edit the stored tensors (so that what random weights would hide shows)."""
    import os

    import carbon_engine_b200.models  # noqa: F401
    from carbon_engine_b200.config.rapovik import RapovikConfig
    from carbon_engine_b200.weights.loader import write_random_model
    out = write_random_model(RapovikConfig.from_dict(dict(raw)), folder, seed=seed)
    path = os.path.join(out, "model.safetensors")
    from helpers import read_raw_safetensors, write_safetensors_plain
    t = read_raw_safetensors(path)
    for name in t:
        # random projections of 0.02 leave the activations' clamps, the gates' caps and the experts' choice untouched
        if name.split(".")[-1] in ("gate", "up", "router", "i", "f", "in") and t[name].dim() == 2:
            t[name] = (t[name].float() * 8.0).to(t[name].dtype)
    if change is not None:
        change(t)
    write_safetensors_plain(path, t)
    return out
