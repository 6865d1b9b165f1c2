"""A recurrent mixer: a matrix memory with exponential gates (mLSTM; Beck et al., "xLSTM: Extended Long
Short-Term Memory", 2024).

With ``h`` the mixer's input and, per head, a memory ``S [dim, vdim]``, a normalizer ``n [dim]`` and a running
maximum ``m``, all zero before a request's first token and 32-bit:

    q, k, v = W_q h / sqrt(dim), W_k h, W_v h
    i = c tanh((W_i h + b_i) / c),   f = log sigmoid(c tanh((W_f h + b_f) / c))        c = gate_cap
    m' = max(f + m, i);   a = f + m - m',   s = i - m'
    S <- exp(a) S + exp(s) k v^T;   n <- exp(a) n + exp(s) k
    o = S^T q / (max(|n . q|, exp(-m')) + 1e-6)
    out = W_o ( rms(o) * w_norm * sigmoid(W_g h) )                      rms per head

``m`` is the same number however the memory is computed (``a``, ``s`` <= 0, so nothing overflows), and once it is
known the memory is a state space with one decay ``exp(a)`` and one step ``exp(s)`` per head and token, and the
normalizer its row with the constant input one: a stretch of tokens runs on the state-space kernels. The
queries, keys and values are rounded to the compute dtype; the gates, ``m``, both decays, ``S``, ``n`` and the
read-out are 32-bit. The state of a request is one row of a fixed-size state array: ``S`` of all heads, each
``[vdim, dim]``, then ``n``, then ``m``.
"""
from __future__ import annotations

import math
from typing import Optional

import torch

from .base import FixedState, Mixer, TensorSpec, register_mixer


@register_mixer("matrix_memory")
class MatrixMemory(Mixer):
    """``names``: the tensors' local names (the gates' biases are their names with ``.b`` added)."""
    graph_safe = True

    def __init__(self, width: int, heads: int, dim: int, vdim: int, gate_cap: float, eps: float, scale: Optional[float] = None,
                 names: Optional[dict] = None, init_std: float = 0.02):
        if not gate_cap > 0:
            raise ValueError(f"gates are capped by a positive number, got {gate_cap}")
        self.width, self.heads, self.dim, self.vdim = int(width), int(heads), int(dim), int(vdim)
        self.gate_cap, self.eps, self.init_std = float(gate_cap), float(eps), float(init_std)
        self.scale = float(scale) if scale is not None else 1.0 / math.sqrt(self.dim)
        self.names = dict({"q": "q", "k": "k", "v": "v", "g": "g", "i": "i", "f": "f", "norm": "norm", "o": "o"}, **(names or {}))
        self.inner, self.key_rows = self.heads * self.vdim, self.heads * self.dim
        self.channels = self.inner + 2 * self.key_rows               # v | k | q
        self.state_floats = self.inner * self.dim + self.key_rows + self.heads

    def tensors(self):
        n, init, vec = self.names, ("normal", self.init_std), dict(role="vector")
        H, d = self.heads, self.width
        return {n["q"]: TensorSpec((self.key_rows, d), init=init), n["k"]: TensorSpec((self.key_rows, d), init=init),
                n["v"]: TensorSpec((self.inner, d), init=init), n["g"]: TensorSpec((self.inner, d), init=init),
                n["i"]: TensorSpec((H, d), init=init), n["i"] + ".b": TensorSpec((H,), init=("normal", 1.0), **vec),
                n["f"]: TensorSpec((H, d), init=init), n["f"] + ".b": TensorSpec((H,), init=("uniform", 1.0, 6.0), **vec),
                n["norm"]: TensorSpec((self.inner,), init=("normal_about_one", 0.1), **vec),
                n["o"]: TensorSpec((d, self.inner), init=init)}

    def cache_need(self):
        return FixedState(((self.state_floats + 3) // 4 * 4,), torch.float32)

    def load(self, tensors, ops, dtype):
        super().load(tensors, ops, dtype)
        n = self.names
        rows = [tensors[n[key]] for key in ("v", "k", "q", "g", "i", "f")]
        pad = -sum(r.shape[0] for r in rows) % 8        # whole groups of eight rows for the tensor-core products
        if pad:
            rows.append(torch.zeros(pad, self.width, dtype=rows[0].dtype, device=rows[0].device))
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_act, self.w_gates = self.w_in[:self.channels], self.w_in[self.channels:]
        self.w_o = tensors[n["o"]].contiguous()
        self.b_i, self.b_f, self.norm_w = (tensors[n[key]].float().contiguous() if key == "norm" else tensors[n[key] + ".b"].float().contiguous()
                                           for key in ("i", "f", "norm"))

    def forward(self, ctx, h, cache, residual=None):
        ops, ws = self.ops, ctx.ws
        T, C = h.shape[0], self.channels
        if ctx.batch.max_q_len == 1:          # single tokens: one product; the recurrence rounds what it reads
            proj = ws.get("memory_proj", (T, self.w_in.shape[0]), torch.float32)
            ops.linear(h, self.w_in, proj)
            act, gates = proj[:, :C], proj[:, C:]
        else:
            act = ws.get("memory_act", (T, C), self.dtype)
            gates = ws.get("memory_gates", (T, self.w_gates.shape[0]), torch.float32)
            ops.linear(h, self.w_act, act)
            ops.linear(h, self.w_gates, gates)
        out = ws.get("memory_out", (T, self.inner), self.dtype)
        ops.matrix_memory(ctx, act, gates, self.b_i, self.b_f, self.gate_cap, self.norm_w, self.scale, self.eps, cache.state,
                          self.heads, self.dim, self.vdim, out)
        if residual is not None:
            ops.linear(out, self.w_o, residual, accumulate=True)
            return None
        y = ws.get("mixer_out", (T, self.width), torch.float32)
        ops.linear(out, self.w_o, y)
        return y
