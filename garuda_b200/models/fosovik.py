"""The Fosovik decoder as a ``ModelSpec``.

An embedding times a constant; layers that have one norm, whose output both sublayers read: ``x <- x +
mixer(h) + ff(h)`` with ``h = norm(x)``; the norm is ``tanh(alpha x) w + b``, without a mean or a variance.
A layer's mixer is one of two: attention without a position encoding, whose queries and keys are divided
by their root mean square per head (no weight), whose queries grow with the logarithm of their position,
with a learned sink per head, and which may read the keys and values of an earlier layer instead of having
its own; or a state-space recurrence (Mamba-2). The feed-forward is a clamped gated one or routed experts
``down(gelu(up h))`` weighed by their share of a softmax over all experts, or absent. A final norm of the
same kind; a head of its own.
Tensor names: ``embed``, ``head``, ``final.norm``, and per layer ``l<i>.norm1``, ``l<i>.mix.*``,
``l<i>.mlp.*``; a norm's other tensors are its name with ``.alpha`` and ``.b`` added.
"""
from __future__ import annotations

from ..config.fosovik_config import FosovikConfig
from ..config.registry import register_architecture
from ..parts.base import PartSpec
from ..parts.block import BlockSpec
from .decoder import ModelSpec, LayerCall


def _norm(cfg, prefix, name):
    return PartSpec("dynamic_tanh", dict(width=cfg.width, weight_name=name), prefix=prefix)


def _mixer(cfg, layer, p):
    m = layer.mixer
    if layer.type == "mamba2":
        return PartSpec("state_space_duality", dict(
            width=cfg.width, heads=m.heads, groups=m.groups, state=m.state, vdim=m.vdim, taps=m.taps,
            norm_groups=m.norm_groups, eps=cfg.eps), prefix=p)
    return PartSpec("normed_key_attention", dict(
        width=cfg.width, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, qk_norm=True,
        qk_norm_weight=False, eps=cfg.eps, temperature=False, values="projected", gate=False, sink=True,
        query_growth=m.q_temp, reads_shared_cache=m.kv_from is not None), prefix=p)


def _feed_forward(cfg, f, p):
    if f is None:
        return None
    if f.kind == "dense":
        return PartSpec("gated", dict(width=cfg.width, inner=f.ff, activation="clamped_swish", limit=f.limit), prefix=p)
    return PartSpec("routed_experts", dict(width=cfg.width, experts=f.experts, top=f.top, inner=f.ff, gated=False,
                                           activation="gelu", router_bias=False, router_score="softmax_all"), prefix=p)


def fosovik_spec(cfg: FosovikConfig) -> ModelSpec:
    layers, order = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        layers.append(BlockSpec(mixer=_mixer(cfg, layer, p + "mix."), feed_forward=_feed_forward(cfg, layer.mlp, p + "mlp."),
                                mixer_norm=_norm(cfg, p, "norm1"), feed_forward_norm=None, arrangement="parallel"))
        # a layer is run once and in its place, so a layer's number is also its entry in the run order
        order.append(LayerCall(i, reads_cache_of=layer.mixer.kv_from if layer.type == "attention" else None))
    return ModelSpec(
        architecture=cfg.architecture, width=cfg.width, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding="embed", layers=layers, order=order, final_norm=_norm(cfg, "", "final.norm"), head="head",
        embedding_scale=cfg.embedding_scale, eos_token_ids=cfg.eos_token_ids)


register_architecture("Fosovik", FosovikConfig.from_dict, fosovik_spec)
