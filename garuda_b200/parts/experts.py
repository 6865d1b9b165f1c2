"""A feed-forward of routed experts: a router picks ``top`` of ``experts`` small
gated feed-forwards per token, their outputs are summed with the router's
weights, and an optional shared expert runs for every token.

    z      = W_r h + b_r                      (32-bit)
    chosen = the ``top`` largest z, weights = softmax over the chosen z only
    expert(h) = W_down act(W_gate h, W_up h)  (``act`` as in ``GatedFeedForward``)
    out    = sum_chosen weight_e * expert_e(h) + shared(h)

Variants, by constructor parameter: ``router_score="sigmoid"`` weighs a chosen expert by
``sigmoid(z_e)`` (the choice is still of the largest; nothing is renormalized);
``router_score="softmax_all"`` weighs it by its share of the softmax over all experts' logits
(not renormalized over the chosen either);
``scale_input=True`` puts the weight on what goes into the expert, ``out = sum_chosen
expert_e(weight_e * h)``; ``router_bias=False`` drops ``b_r``; ``activation="silu"`` is the plain
SiLU gate; ``gated=False`` makes an expert ``W_down act(W_up h)`` without a gate (``activation`` = ``"gelu"``,
the exact one, or any activation of ``PlainFeedForward`` without numbers of its own).

How the experts are chosen: ``correction=True`` adds a learned number per expert to the scores for the choice
alone (``router_score`` = ``"sigmoid"`` or ``"softmax_all"``; the weights stay the scores without it).
``groups=(count, keep)`` forms equal groups of neighbours, a group's score being its best expert's, and only the
``keep`` best groups' experts can be chosen. ``identity=n``: the router's last ``n`` outputs are experts without tensors that
return their input.

Tensor names: ``router``, ``router.b``, ``correction``, ``e<i>.gate|up|down`` (no ``gate`` without one), ``shared.gate|up|down``.
"""
from __future__ import annotations

from typing import Optional

import torch

from .base import FeedForward, TensorSpec, register_feed_forward

#: activations of one value that the expert and the plain feed-forward kernels know
PLAIN_ACTIVATIONS = ("relu2", "silu", "tanh", "sigmoid", "gelu")


@register_feed_forward("routed_experts")
class RoutedExperts(FeedForward):
    graph_safe = True
    scales_residual = True

    def __init__(self, width: int, experts: int, top: int, inner: int, activation: str = "clamped_swish",
                 limit: float = 0.0, shared_inner: Optional[int] = None, shared_limit: float = 0.0,
                 router_bias: bool = True, init_std: float = 0.02, router_score: str = "softmax_chosen",
                 scale_input: bool = False, gated: bool = True, correction: bool = False, identity: int = 0, groups=None):
        if not gated and (shared_inner or activation not in PLAIN_ACTIVATIONS):
            raise ValueError(f"experts without a gate take {PLAIN_ACTIVATIONS} and no shared expert, got {activation!r}")
        self.gated = bool(gated)
        if router_score not in ("softmax_chosen", "sigmoid", "softmax_all"):
            raise ValueError(f"unknown router score {router_score!r}")
        self.router_score, self.scale_input = router_score, bool(scale_input)
        self.identity, self.correction = int(identity), bool(correction)
        self.choices = int(experts) + self.identity              # the router's outputs
        self.groups = (int(groups[0]), int(groups[1])) if groups is not None and int(groups[1]) < int(groups[0]) else None
        if self.groups and (self.groups[1] < 1 or self.choices % self.groups[0]):
            raise ValueError(f"{self.choices} experts do not form {self.groups[0]} equal groups of which {self.groups[1]} are kept")
        within = self.choices if not self.groups else self.choices // self.groups[0] * self.groups[1]
        if not 1 <= top <= within:
            raise ValueError(f"a token uses 1 to {within} experts, got {top}")
        if self.correction and router_score == "softmax_chosen":
            raise ValueError("a correction of the scores goes with scores that do not depend on the choice")
        if self.identity and self.scale_input:
            raise ValueError("experts that return their input have their weight on what they return")
        self.width, self.experts, self.top, self.inner = int(width), int(experts), int(top), int(inner)
        self.activation, self.limit = activation, float(limit)
        self.shared_inner = int(shared_inner) if shared_inner else None
        self.shared_limit = float(shared_limit)
        self.router_bias = bool(router_bias)
        self.init_std = float(init_std)

    def tensors(self):
        init = ("normal", self.init_std)
        t = {"router": TensorSpec((self.choices, self.width), init=init)}
        if self.router_bias:
            t["router.b"] = TensorSpec((self.choices,), role="vector", init=("normal", 0.02))
        if self.correction:
            t["correction"] = TensorSpec((self.choices,), role="vector", init=("normal", 0.1))
        for e in range(self.experts):
            if self.gated:
                t[f"e{e}.gate"] = TensorSpec((self.inner, self.width), init=init)
            t[f"e{e}.up"] = TensorSpec((self.inner, self.width), init=init)
            t[f"e{e}.down"] = TensorSpec((self.width, self.inner), init=init)
        if self.shared_inner:
            t["shared.gate"] = TensorSpec((self.shared_inner, self.width), init=init)
            t["shared.up"] = TensorSpec((self.shared_inner, self.width), init=init)
            t["shared.down"] = TensorSpec((self.width, self.shared_inner), init=init)
        return t

    def load(self, tensors, ops, dtype):
        super().load(tensors, ops, dtype)
        self.w_router = tensors["router"].contiguous()
        self.b_router = tensors["router.b"].float().contiguous() if self.router_bias else None
        self.choice = {}                  # what the router is told about the choice, beyond the logits
        if self.correction:
            self.choice["correction"] = tensors["correction"].float().contiguous()
        if self.groups:
            self.choice["groups"] = self.groups
        E = self.experts
        # the experts' gate and up rows stacked in the kernels' layout, or the up rows alone; [E, width, inner]
        if self.gated:
            self.w_gate_up = ops.pack_expert_gate_up([tensors[f"e{e}.gate"] for e in range(E)],
                                                     [tensors[f"e{e}.up"] for e in range(E)])
        else:
            self.w_gate_up = torch.stack([tensors[f"e{e}.up"] for e in range(E)]).contiguous()
        self.w_down = torch.stack([tensors[f"e{e}.down"] for e in range(E)]).contiguous()
        if self.shared_inner:
            self.w_shared_gate_up = ops.pack_gate_up(tensors["shared.gate"], tensors["shared.up"])
            self.w_shared_down = tensors["shared.down"].contiguous()

    @property
    def emits_tanh_norm(self):
        """Whether ``forward`` takes ``emit_norm``, a ``DynamicTanh`` of the residual that this part is the last to write."""
        return not self.shared_inner

    #: ``forward`` takes ``leave_rows``: the output may be left as rows that the pass behind adds up
    leaves_rows = True

    def forward(self, ctx, h, residual=None, alpha: float = 1.0, emit_norm=None, leave_rows: bool = False):
        ops, ws = self.ops, ctx.ws
        T = h.shape[0]
        target = residual
        shared_first = target is None and self.shared_inner
        leave_rows = leave_rows and self.gated and not self.scale_input and getattr(ops, "leaves_expert_rows", False)
        if target is None:
            target = ws.get("ffn_out", (T, self.width), torch.float32)
            alpha = 1.0
            if shared_first:
                self._shared(ctx, h, target, accumulate=False)       # stored: the routed ones are added to it
            elif not leave_rows:
                target.zero_()
        ids = ws.get("expert_ids", (T, self.top), torch.int32)
        weights = ws.get("expert_weights", (T, self.top), torch.float32)
        if leave_rows and residual is None:
            ops.route_topk(h, self.w_router, self.b_router, self.top, ids, weights, score=self.router_score, **self.choice)
            rows = ops.expert_rows(ctx, h, self.w_gate_up, self.w_down, ids, weights, self.activation, self.limit,
                                   identity=bool(self.identity), base=target if shared_first else None)
            if rows is not None:
                return rows
            if not shared_first:
                target.zero_()
            ops.routed_feed_forward(ctx, h, self.w_gate_up, self.w_down, ids, weights, target, self.activation, self.limit,
                                    identity=bool(self.identity))
            return target
        if self.router_score == "softmax_chosen" and not self.scale_input and self.gated and not self.choice and not self.identity:
            ops.route_topk(h, self.w_router, self.b_router, self.top, ids, weights)
            ops.routed_feed_forward(ctx, h, self.w_gate_up, self.w_down, ids, weights, target, self.activation,
                                    self.limit, alpha)
        else:
            ops.route_topk(h, self.w_router, self.b_router, self.top, ids, weights, score=self.router_score, **self.choice)
            kw = {} if self.gated else {"gated": False}
            if self.identity:
                kw["identity"] = True
            if emit_norm is not None and residual is not None:
                turn = ctx.step_cache["tanh_turn"] = ctx.step_cache.get("tanh_turn", 0) ^ 1       # the norm in front may still be read
                kw["then"] = (emit_norm.alpha, emit_norm.weight, emit_norm.bias,
                              ws.get(f"tanh_normed_{turn}", (T, self.width), torch.bfloat16))
            emitted = ops.routed_feed_forward(ctx, h, self.w_gate_up, self.w_down, ids, weights, target, self.activation,
                                              self.limit, alpha, scale_input=self.scale_input, **kw)
            if emitted:
                ctx.pending_norm = kw["then"][3]
        if self.shared_inner and not shared_first:
            self._shared(ctx, h, target, accumulate=True, alpha=alpha)
        return None if residual is not None else target

    def _shared(self, ctx, h, target, **kw):
        act = ctx.ws.get("shared_act", (h.shape[0], self.shared_inner), self.dtype)
        self.ops.linear_gated(ctx, h, self.w_shared_gate_up, act, self.activation, self.shared_limit)
        self.ops.linear(act, self.w_shared_down, target, **kw)
