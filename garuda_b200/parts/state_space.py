"""A recurrent mixer: the selective state space with one decay per head and token (Mamba-2; Dao and Gu,
"Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State Space
Duality", 2024).

With ``h`` the mixer's input, ``H`` heads of ``vdim`` channels (``inner = H vdim``) that each keep a state
``S [state, vdim]`` per request (32-bit, zero at the start), and ``G`` groups of heads that share the
vectors ``B`` and ``C`` (head ``n`` belongs to group ``n // (H / G)``):

    [z | x | B | C | d] = W_in h                    inner, inner, G state, G state, H
    x, B, C each pass a causal convolution over time per channel (``taps`` taps, the last one on the
    current token, a bias, zeros before the sequence) and SiLU
    dt = softplus(d + dt_bias);   a = exp(-exp(A_log) dt)            per head and token
    S <- a S + dt B x^T;   y = S^T C + D x                           per head and token
    out = W_o ( rms(y * silu(z)) * w_norm )       the mean square over each of ``norm_groups`` equal parts

Step sizes, decays, the state and everything between them are 32-bit; the convolved activations are
rounded to the compute dtype, as operands of the products that the recurrence over a stretch of tokens
amounts to. The state of a request is one row of a fixed-size state array: ``S`` of all heads, each
``[vdim, state]``, then the convolution's last ``taps - 1`` inputs.
"""
from __future__ import annotations

from typing import Optional

import torch

from .base import FixedState, Mixer, TensorSpec, register_mixer


@register_mixer("state_space_duality")
class StateSpaceDuality(Mixer):
    """``names``: the tensors' local names (the convolution's bias is its name with ``.b`` added;
    ``conv_bias=False``: none)."""
    graph_safe = True
    scales_residual = True

    def __init__(self, width: int, heads: int, groups: int, state: int, vdim: int, taps: int, eps: float,
                 norm_groups: int = 1, conv_bias: bool = True, names: Optional[dict] = None, init_std: float = 0.02):
        if heads % groups:
            raise ValueError(f"{heads} heads are not a multiple of {groups} groups")
        if heads * vdim % norm_groups:
            raise ValueError(f"{heads * vdim} channels do not split into {norm_groups} equal parts")
        if taps < 1:
            raise ValueError(f"the convolution needs at least one tap, got {taps}")
        self.width, self.heads, self.groups = int(width), int(heads), int(groups)
        self.state, self.vdim, self.taps, self.eps = int(state), int(vdim), int(taps), float(eps)
        self.norm_groups, self.conv_bias, self.init_std = int(norm_groups), bool(conv_bias), float(init_std)
        self.names = dict({"in": "in", "conv": "conv", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D", "norm": "norm",
                           "o": "o"}, **(names or {}))
        self.inner = self.heads * self.vdim
        self.channels = self.inner + 2 * self.groups * self.state
        self.rows = self.inner + self.channels + self.heads

    def tensors(self):
        n, vec = self.names, dict(role="vector")
        t = {n["in"]: TensorSpec((self.rows, self.width), init=("normal", self.init_std)),
             n["conv"]: TensorSpec((self.channels, self.taps), init=("normal", 0.4), **vec),
             n["dt_bias"]: TensorSpec((self.heads,), init=("uniform", -3.0, 0.5), **vec),
             n["A_log"]: TensorSpec((self.heads,), init=("uniform", -2.0, 2.0), **vec),
             n["D"]: TensorSpec((self.heads,), init=("normal_about_one", 0.3), **vec),
             n["norm"]: TensorSpec((self.inner,), init=("normal_about_one", 0.1), **vec),
             n["o"]: TensorSpec((self.width, self.inner), init=("normal", self.init_std))}
        if self.conv_bias:
            t[n["conv"] + ".b"] = TensorSpec((self.channels,), init=("normal", 0.1), **vec)
        return t

    def cache_need(self):
        return FixedState((self.inner * self.state + (self.taps - 1) * self.channels,), torch.float32)

    def load(self, tensors, ops, dtype):
        super().load(tensors, ops, dtype)
        n, vec = self.names, torch.float32
        w = tensors[n["in"]]
        pad = (-self.rows) % 8            # whole groups of eight rows for the tensor-core products
        if pad:
            w = torch.cat([w, torch.zeros(pad, self.width, dtype=w.dtype, device=w.device)], dim=0)
        self.w_in = w.contiguous()
        self.w_o = tensors[n["o"]].contiguous()
        self.conv_w = tensors[n["conv"]].to(vec).contiguous()
        self.conv_b = tensors[n["conv"] + ".b"].to(vec).contiguous() if self.conv_bias else None
        self.dt_bias = tensors[n["dt_bias"]].to(vec).contiguous()
        self.rate = torch.exp(tensors[n["A_log"]].double()).to(vec).contiguous()        # exp(A_log), rounded once
        self.skip = tensors[n["D"]].to(vec).contiguous()
        self.norm_w = tensors[n["norm"]].to(vec).contiguous()

    def forward(self, ctx, h, cache, residual=None, alpha: float = 1.0):
        ops, ws = self.ops, ctx.ws
        T = h.shape[0]
        proj = ws.get("ssd_proj", (T, self.w_in.shape[0]), torch.float32)
        ops.linear(h, self.w_in, proj)
        out = ws.get("ssd_out", (T, self.inner), self.dtype)
        ops.state_space(ctx, proj, (0, self.inner, self.inner + self.channels), self.conv_w, self.conv_b, self.rate,
                        self.dt_bias, self.skip, self.norm_w, self.norm_groups, self.eps, cache.state, self.heads,
                        self.groups, self.state, self.vdim, out)
        if residual is not None:
            ops.linear(out, self.w_o, residual, accumulate=True, alpha=alpha)
            return None
        y = ws.get("mixer_out", (T, self.width), torch.float32)
        ops.linear(out, self.w_o, y)
        return y
