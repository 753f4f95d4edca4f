"""The Rapovik decoder, put together from the package's parts.

Every layer normalises what its sublayers read AND what they return: x += norm1b(mixer(norm1(x))); x += norm2b(ff(norm2(x)))
(``parts/block.py`` ``SandwichNormBlock``), with RMS norms whose stored weights are deviations from 1.  The mixer is, as
config.json lists them, latent attention with a sliding window and an interleaved rotation (``parts/latent_attention.py``), a
state-space mixer (``parts/state_space.py``) or a matrix memory (``parts/matrix_memory.py``).  The feed-forward is gated with the
clamped activation and biases (``parts/mlp.py``), or a mixture of such experts without biases, with sigmoid scores, a correction
for the choice, groups scored by their two best members and a shared expert (``parts/moe.py``), or absent.  A span of layers may
run several times in a row with the same weights: the schedule then names those blocks again, each time with a cache of its own.
Tensor names: ``embed``, ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.gate|up|down`` (+ ``.b``) or
``l<i>.mlp.router|correction``, ``l<i>.mlp.e<j>.gate|up|down``, ``l<i>.mlp.shared.gate|up|down``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from typing import Optional

from ..config.rapovik import LATENT_ATTENTION, MAMBA2, MLSTM, RapovikConfig
from ..config.registry import register_architecture
from ..parts.base import FeedForward
from ..parts.block import SandwichNormBlock
from ..parts.embedding import Embedding, LMHead
from ..parts.model import DecoderModel, LayerCall
from ..parts.registry import build_part

#: the clamped activation's factor inside the sigmoid: part of the design
GLU_ALPHA = 1.702


def _feed_forward(mlp: Optional[dict], width: int, prefix: str) -> Optional[FeedForward]:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return build_part("feed_forward", "gated_mlp", hidden=width, intermediate=mlp["ff"], prefix=prefix, activation="clamped",
                          names=("gate", "up", "down"), bias_names=("gate.b", "up.b", "down.b"), limit=mlp["limit"], alpha=GLU_ALPHA)
    r, groups, shared = mlp["router"], mlp["router"].get("groups") or {}, mlp.get("shared") or {}
    return build_part("feed_forward", "routed_experts", hidden=width, experts=r["experts"], top=r["top"], ff=mlp["expert"]["ff"],
                      prefix=prefix, groups=groups.get("count", 1), keep_groups=groups.get("keep", 1), activation="clamped_glu",
                      shared_ff=shared.get("ff", 0), shared_gate=False, scoring="sigmoid", correction=True, group_score="top2",
                      renormalize=False, limit=mlp["expert"]["limit"], shared_limit=shared.get("limit", 0.0), alpha=GLU_ALPHA)


def build_rapovik(cfg: RapovikConfig, max_positions: int) -> DecoderModel:
    W, eps = cfg.width, cfg.norm_eps
    norm = lambda name: build_part("norm", "rmsnorm", width=W, eps=eps, name=name, unit_offset=True)
    rotations = {}            # one table per (rotated part's size, rotated elements, base)

    def rotation(m: dict):
        key = (m["rot_dim"], m["rot"]["dims"], float(m["rot"]["base"]))
        if key not in rotations:
            rotations[key] = build_part("position", "rotary", head_dim=key[0], theta=key[2], max_positions=max_positions,
                                        rotary_dim=key[1], pairing="interleaved")
        return rotations[key]

    blocks = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}", layer["mixer"]
        if layer["type"] == LATENT_ATTENTION:
            mixer = build_part("mixer", "latent_attention", hidden=W, heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"],
                               vdim=m["vdim"], q_rank=0, kv_rank=m["kv_rank"], prefix=f"{p}.mix", eps=eps, position=rotation(m),
                               scale=m["scale"], window=(m.get("mask") or {}).get("size", 0), gate=None)
        elif layer["type"] == MAMBA2:
            mixer = build_part("mixer", "state_space", hidden=W, heads=m["heads"], vdim=m["vdim"], state=m["state"],
                               groups=m["groups"], taps=m["conv"], prefix=f"{p}.mix", eps=eps, norm_groups=m["norm_groups"])
        else:
            assert layer["type"] == MLSTM
            mixer = build_part("mixer", "matrix_memory", hidden=W, heads=m["heads"], dim=m["dim"], vdim=m["vdim"],
                               gate_cap=m["gate_cap"], prefix=f"{p}.mix", eps=eps)
        ffn = _feed_forward(layer["mlp"], W, f"{p}.mlp")
        around = (norm(f"{p}.norm2"), ffn, norm(f"{p}.norm2b")) if ffn is not None else (None, None, None)
        blocks.append(SandwichNormBlock(W, norm(f"{p}.norm1"), mixer, norm(f"{p}.norm1b"), *around))
    schedule = [LayerCall(block, run, True) for run, block in enumerate(cfg.layer_runs())]
    embedding = Embedding(cfg.vocab_size, W, "embed")
    head = LMHead(cfg.vocab_size, W, norm("final.norm"), "head")
    return DecoderModel(cfg, embedding, blocks, head, schedule=schedule)


register_architecture("Rapovik", RapovikConfig.from_dict, build_rapovik, model_types=("rapovik",), replace=True)
