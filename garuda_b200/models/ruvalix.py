"""The Ruvalix decoder as a ``ModelSpec``.

An embedding that is RMS-normed; layers with a norm in front of and behind each sublayer, ``x <- x +
norm_b(sublayer(norm(x)))``, all norms RMS norms whose weight is stored about zero. A layer's mixer is one of
two: differential attention (two softmax maps per head over the same values, the second taken off the first;
queries and keys with biases, RMS-normed per head and map, rotated on their first channels at stretched
frequencies; a sliding window; a gate per head) or a matrix memory with exponential gates (mLSTM). The
feed-forward is a set of routed experts, some of which return their input, chosen within the best groups by
corrected scores, beside a shared expert; or absent. A stretch of the layers may run several times in a row
with the same weights: before every pass the stream is replaced by a linear map of itself and the embedding's
output, and a row of a learned table is added. A final norm; a head of its own.
Tensor names: ``embed``, ``embed.norm``, ``head``, ``final.norm``, ``loop.in``, ``loop.step``, and per layer
``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.*``.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.ruvalix_config import RuvalixConfig
from ..parts.base import PartSpec, TensorSpec
from ..parts.block import BlockSpec
from .decoder import LayerCall, ModelSpec

MIX_MATRIX, STEP_TABLE = "loop.in", "loop.step"


def _norm(cfg, prefix, name):
    return PartSpec("rms", dict(width=cfg.width, eps=cfg.eps, weight_name=name, unit_offset=True), prefix=prefix)


def _mixer(cfg, layer, p):
    m = layer.mixer
    if layer.type == "mlstm":
        return PartSpec("matrix_memory", dict(width=cfg.width, heads=m.heads, dim=m.dim, vdim=m.vdim, gate_cap=m.gate_cap,
                                              eps=cfg.eps), prefix=p)
    scaling = None
    if m.rot_scaling is not None:
        s = m.rot_scaling
        scaling = dict(factor=s.factor, original=s.original, fast=s.fast, slow=s.slow)
    return PartSpec("differential_attention", dict(
        width=cfg.width, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, diff=m.diff, eps=cfg.eps,
        window=m.window, rot_base=m.rot_base, rot_dims=m.rot_dims, rot_scaling=scaling, bias=True, gate=True), prefix=p)


def _feed_forward(cfg, f, p):
    return PartSpec("routed_experts", dict(
        width=cfg.width, experts=f.experts, top=f.top, inner=f.ff, activation="silu", shared_inner=f.shared_ff, router_bias=False,
        router_score="softmax_all", correction=True, identity=f.identity, groups=f.groups), prefix=p)


def ruvalix_spec(cfg: RuvalixConfig) -> ModelSpec:
    layers, ignored, n = [], [], len(cfg.layers)
    for i, layer in enumerate(cfg.layers):
        p, ff = f"l{i}.", layer.mlp is not None
        if not ff:
            ignored += [p + "norm2", p + "norm2b"]           # (a folder may carry them for a layer without a feed-forward)
        layers.append(BlockSpec(
            mixer=_mixer(cfg, layer, p + "mix."), feed_forward=_feed_forward(cfg, layer.mlp, p + "mlp.") if ff else None,
            mixer_norm=_norm(cfg, p, "norm1"), mixer_post_norm=_norm(cfg, p, "norm1b"),
            feed_forward_norm=_norm(cfg, p, "norm2") if ff else None,
            feed_forward_post_norm=_norm(cfg, p, "norm2b") if ff else None, arrangement="sandwich_norm"))
    order, extra = [LayerCall(i) for i in range(n)], {}
    if cfg.loop is not None:
        start, stop, times = cfg.loop
        order = [LayerCall(i) for i in range(start)]
        for t in range(times):
            for i in range(start, stop):
                first = i == start
                order.append(LayerCall(i, mix_embedding=MIX_MATRIX if first else None, add_row=(STEP_TABLE, t) if first else None))
        order += [LayerCall(i) for i in range(stop, n)]
        extra = {MIX_MATRIX: TensorSpec((cfg.width, 2 * cfg.width)),
                 STEP_TABLE: TensorSpec((times, cfg.width), role="vector", init=("normal", 0.1))}
    else:
        ignored += [MIX_MATRIX, STEP_TABLE]
    return ModelSpec(
        architecture=cfg.architecture, width=cfg.width, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding="embed", embedding_norm=_norm(cfg, "", "embed.norm"), layers=layers, order=order,
        final_norm=_norm(cfg, "", "final.norm"), head="head", extra_tensors=extra or None, eos_token_ids=cfg.eos_token_ids,
        ignored_tensors=tuple(ignored))


register_architecture("Ruvalix", RuvalixConfig.from_dict, ruvalix_spec)
