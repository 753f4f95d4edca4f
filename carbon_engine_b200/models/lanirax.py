"""The Lanirax decoder, put together from the package's parts.

The norm sits behind the sum and is the new residual: x <- norm1(alpha x + mixer(x)), x <- norm2(alpha x + ff(x))
(``parts/block.py`` ``PostNormBlock``), with RMS norms; the embedding is normed too.  The mixer is, as config.json lists them,
softmax attention without a rotation, with a query temperature that grows with the position and a penalty per head that grows
with a key's distance (``parts/sink_attention.py``), or two mixers side by side whose outputs are normed over the width and added
with the factor 1/2 (``parts/combine.py`` ``NormedMixers``): windowed attention whose values are the projected keys, with a
stretched rotation of neighbouring pairs, a norm behind the rotation and a sink per head (``parts/sink_attention.py``), beside the
gated delta rule with one decay per head (``parts/gated_delta.py`` ``HeadGatedDelta``).  The feed-forward is a mixture of gated
SiLU experts weighted by a softmax over the chosen logits (``parts/moe.py``), or absent.  A layer may run another layer's weights
with a cache of its own, which the model's schedule expresses as a second call of that layer's block.
Tensor names: ``embed``, ``embed.norm``, ``l<i>.norm1|norm2``, ``l<i>.mix.*`` (``.left.*`` and ``.right.*`` for the pair, with
``.left.out`` and ``.right.out``), ``l<i>.mlp.router`` (+ ``.b``), ``l<i>.mlp.e<j>.gate|up|down``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import math

from ..config.lanirax import ATTENTION, PARALLEL, LaniraxConfig, weight_owner
from ..config.registry import register_architecture
from ..parts.block import PostNormBlock
from ..parts.embedding import Embedding, LMHead
from ..parts.model import DecoderModel, LayerCall
from ..parts.registry import build_part
from ..parts.rope import QueryTemperature, RopeScaling


def distance_slopes(heads: int):
    """What a token of distance costs, per head: 2^(-8 (h + 1) / heads), h from 0."""
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def build_lanirax(cfg: LaniraxConfig, max_positions: int) -> DecoderModel:
    W, eps = cfg.width, cfg.norm_eps
    norm = lambda name: build_part("norm", "rmsnorm", width=W, eps=eps, name=name)
    rotations, temperatures = {}, {}            # one table per distinct set of constants

    def rotation(m: dict):
        rot = m.get("rot")
        if not rot:
            return None
        s = rot.get("scaling")
        key = (m["dim"], rot["dims"], float(rot["base"]), tuple(float(s[k]) for k in ("factor", "original", "fast", "slow")) if s else None)
        if key not in rotations:
            scaling = None
            if s:
                factor, original, fast, slow = key[3]
                scaling = RopeScaling("yarn", factor=factor, original_max_position=original, beta_fast=fast, beta_slow=slow,
                                      attention_factor=0.1 * math.log(factor) + 1.0)
            rotations[key] = build_part("position", "rotary", head_dim=key[0], theta=key[2], max_positions=max_positions,
                                        rotary_dim=key[1], scaling=scaling, pairing="interleaved")
        return rotations[key]

    def temperature(m: dict):
        t = m.get("q_temp")
        if not t:
            return None
        key = (float(t["coef"]), float(t["every"]))
        if key not in temperatures:
            temperatures[key] = QueryTemperature(*key, max_positions=max_positions)
        return temperatures[key]

    def pair(m: dict, prefix: str):
        left, right = m["left"], m["right"]
        attention = build_part("mixer", "sink_attention", hidden=W, heads=left["heads"], kv_heads=left["kv_heads"], dim=left["dim"],
                               prefix=f"{prefix}.left", eps=eps, position=rotation(left), scale=left["scale"],
                               window=(left.get("mask") or {}).get("size", 0), qk_norm="after_plain", tied_values=True, sink=True)
        delta = build_part("mixer", "head_gated_delta", hidden=W, heads=right["heads"], kv_heads=right["kv_heads"], dim=right["dim"],
                           vdim=right["vdim"], taps=right["conv"], prefix=f"{prefix}.right", eps=eps, gate="silu")
        return build_part("mixer", "normed_mixers", members=[attention, delta],
                          norms=[norm(f"{prefix}.left.out"), norm(f"{prefix}.right.out")], factor=0.5)

    blocks, block_of = [], {}
    for i, layer in enumerate(cfg.layers):
        if layer.get("weights_of") is not None:
            continue
        p, m, mlp = f"l{i}", layer["mixer"], layer["mlp"]
        if layer["type"] == ATTENTION:
            mixer = build_part("mixer", "sink_attention", hidden=W, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"],
                               vdim=m["vdim"], prefix=f"{p}.mix", eps=eps, scale=m["scale"], qk_norm="before",
                               query_temperature=temperature(m), distance_slopes=distance_slopes(m["heads"]))
        else:
            assert layer["type"] == PARALLEL
            mixer = pair(m, f"{p}.mix")
        ffn = ffn_norm = None
        if mlp is not None:
            ffn_norm = norm(f"{p}.norm2")
            ffn = build_part("feed_forward", "routed_experts", hidden=W, experts=mlp["router"]["experts"], top=mlp["router"]["top"],
                             ff=mlp["expert"]["ff"], prefix=f"{p}.mlp", activation="silu_glu", scoring="softmax_chosen", router_bias=True)
        block_of[i] = len(blocks)
        blocks.append(PostNormBlock(W, cfg.alpha, mixer, norm(f"{p}.norm1"), ffn, ffn_norm))
    schedule = [LayerCall(block_of[weight_owner(cfg.layers, i)], i, True) for i in range(len(cfg.layers))]
    embedding = Embedding(cfg.vocab_size, W, "embed", norm=norm("embed.norm"), leave_rounded=True)
    head = LMHead(cfg.vocab_size, W, norm("final.norm"), "head")
    return DecoderModel(cfg, embedding, blocks, head, schedule=schedule)


register_architecture("Lanirax", LaniraxConfig.from_dict, build_lanirax, model_types=("lanirax",), replace=True)
