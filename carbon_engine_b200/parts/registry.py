"""Registries of part kinds, so that a configuration can choose each layer's mixer, feed-forward,
norm and position encoding by name, and so that new kinds can be added from outside the package.

A factory takes keyword parameters (sizes, constants, the tensor-name prefix) and returns the part.
"""
from __future__ import annotations

from typing import Callable, Dict

from .attention import PagedAttention
from .delta_rule import GeneralDeltaRule
from .diff_attention import DifferentialAttention
from .combine import NormedMixers, SummedMixers
from .gated_delta import ChannelGatedDelta, HeadGatedDelta
from .latent_attention import LatentAttention
from .masked_attention import GatedWindowAttention
from .matrix_memory import MatrixMemory
from .mlp import DenseMLP, GatedMLP
from .moe import RoutedExperts
from .norm import GroupedRMSNorm, LayerNorm, RMSNorm
from .retention import Retention
from .rope import NoPositionEncoding, RotaryEmbedding
from .sink_attention import SinkAttention
from .state_space import StateSpace

_KINDS: Dict[str, Dict[str, Callable]] = {"mixer": {}, "feed_forward": {}, "norm": {}, "position": {}}


def register_part(kind: str, name: str, factory: Callable, replace: bool = False) -> None:
    table = _KINDS[kind]
    if name in table and not replace:
        raise ValueError(f"{kind} '{name}' is already registered")
    table[name] = factory


def unregister_part(kind: str, name: str) -> None:
    _KINDS[kind].pop(name, None)


def build_part(kind: str, part: str, /, **params):
    try:
        factory = _KINDS[kind][part]
    except KeyError:
        raise ValueError(f"unknown {kind} '{part}' (registered: {', '.join(sorted(_KINDS[kind]))})") from None
    return factory(**params)


def register_mixer(name, factory, replace=False): register_part("mixer", name, factory, replace)
def register_feed_forward(name, factory, replace=False): register_part("feed_forward", name, factory, replace)
def register_norm(name, factory, replace=False): register_part("norm", name, factory, replace)
def register_position(name, factory, replace=False): register_part("position", name, factory, replace)


register_mixer("full_attention", lambda **kw: PagedAttention(**{**kw, "window": 0}))
register_mixer("sliding_attention", lambda **kw: PagedAttention(**kw))
register_mixer("differential_attention", DifferentialAttention)
register_mixer("general_delta", GeneralDeltaRule)
register_mixer("gated_window_attention", GatedWindowAttention)
register_mixer("latent_attention", LatentAttention)
register_mixer("channel_gated_delta", ChannelGatedDelta)
register_mixer("head_gated_delta", HeadGatedDelta)
register_mixer("retention", Retention)
register_mixer("sink_attention", SinkAttention)
register_mixer("summed_mixers", SummedMixers)
register_mixer("normed_mixers", NormedMixers)
register_mixer("state_space", StateSpace)
register_mixer("matrix_memory", MatrixMemory)
register_feed_forward("gated_mlp", GatedMLP)
register_feed_forward("dense_mlp", DenseMLP)
register_feed_forward("routed_experts", RoutedExperts)
register_norm("rmsnorm", RMSNorm)
register_norm("grouped_rmsnorm", GroupedRMSNorm)
register_norm("layernorm", LayerNorm)
register_position("rotary", RotaryEmbedding)
register_position("none", lambda **kw: NoPositionEncoding())
