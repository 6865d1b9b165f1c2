"""Differential attention over the paged cache (Ye et al., "Differential Transformer", 2024): every head has two
softmax maps over the same values, and the second, times a learned number, is taken off the first.

With ``h`` the mixer's input, query head ``n`` reading key/value head ``g = n // (heads / kv_heads)``, map ``r`` = 1, 2:

    q^r_n, k^r_g = W_q h + b_q, W_k h + b_k       (``dim`` channels per head and map);   v_g = W_v h + b_v   (``vdim``)
    q, k <- rms(q) * w_q, rms(k) * w_k             per head and map; the weights shared by all of them
    q, k rotated at their positions on their first ``rot_dims`` channels: channel i with i + rot_dims / 2
    p^r_ij = softmax over the keys with 0 <= i - j < window of (q^r_i . k^r_j) * scale
    o = sum_j (p^1_ij - lambda p^2_ij) v_j,  lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff
    out = W_o concat_n ( rms(o) * (1 - diff) * sigmoid(W_g h)_n )                     rms per head, no weight

A cached key row holds both maps' keys of a key head side by side, and its value once: a tile of keys and
values is read once for both maps, and the difference, its norm and the gate are the attention kernel's epilogue
(the two maps are never rounded before they are subtracted).
"""
from __future__ import annotations

import math
from typing import Optional

import torch

from .base import Mixer, PagedKV, TensorSpec, register_mixer
from .rotary import Rotary

MAPS = 2


@register_mixer("differential_attention")
class DifferentialAttention(Mixer):
    """``names``: the tensors' local names (a bias is the weight's name with ``.b`` added). ``rot_base`` None: not
    rotated; ``rot_scaling``: see ``rotary.stretched_frequencies``. ``bias``, ``qk_norm``, ``gate``: leave out what they name."""
    graph_safe = True

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: Optional[int] = None, scale: Optional[float] = None,
                 diff: float = 0.8, eps: float = 1e-6, window: Optional[int] = None, rot_base: Optional[float] = None,
                 rot_dims: int = 0, rot_layout: str = "half", rot_scaling: Optional[dict] = None, qk_norm: bool = True,
                 bias: bool = False, gate: bool = False, names: Optional[dict] = None, init_std: float = 0.02):
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads are not a multiple of {kv_heads} kv heads")
        self.width, self.heads, self.kv_heads, self.dim = int(width), int(heads), int(kv_heads), int(dim)
        self.vdim = int(vdim) if vdim else MAPS * self.dim
        self.scale = float(scale) if scale is not None else 1.0 / math.sqrt(self.dim)
        self.diff, self.eps, self.window = float(diff), float(eps), int(window) if window else None
        self.qk_norm, self.bias, self.gate, self.init_std = bool(qk_norm), bool(bias), bool(gate), float(init_std)
        self.names = dict({"q": "q", "k": "k", "v": "v", "o": "o", "g": "g", "q_norm": "q.norm", "k_norm": "k.norm", "lq1": "lq1",
                           "lk1": "lk1", "lq2": "lq2", "lk2": "lk2"}, **(names or {}))
        self.rotary = None
        if rot_base is not None and rot_dims:
            self.rotary = Rotary(float(rot_base), int(rot_dims), layout=rot_layout, scaling=rot_scaling or {"factor": 1.0}).rotary
        self.q_dim, self.k_dim = MAPS * self.heads * self.dim, MAPS * self.kv_heads * self.dim
        self.v_dim, self.ctx_dim = self.kv_heads * self.vdim, self.heads * self.vdim

    def tensors(self):
        init, n, vec = ("normal", self.init_std), self.names, dict(role="vector")
        t = {n["q"]: TensorSpec((self.q_dim, self.width), init=init), n["k"]: TensorSpec((self.k_dim, self.width), init=init),
             n["v"]: TensorSpec((self.v_dim, self.width), init=init), n["o"]: TensorSpec((self.width, self.ctx_dim), init=init)}
        if self.bias:
            for key, rows in (("q", self.q_dim), ("k", self.k_dim), ("v", self.v_dim)):
                t[n[key] + ".b"] = TensorSpec((rows,), init=("normal", 0.1), **vec)
        if self.qk_norm:
            for key in ("q_norm", "k_norm"):
                t[n[key]] = TensorSpec((self.dim,), init=("normal_about_one", 0.1), **vec)
        for key in ("lq1", "lk1", "lq2", "lk2"):
            t[n[key]] = TensorSpec((self.dim,), init=("normal", 0.1), **vec)
        if self.gate:
            t[n["g"]] = TensorSpec((self.heads, self.width), init=init)
        return t

    def cache_need(self):
        return PagedKV(self.kv_heads, MAPS * self.dim, self.window, value_dim=self.vdim)

    def load(self, tensors, ops, dtype):
        super().load(tensors, ops, dtype)
        n = self.names
        rows = [tensors[n[key]] for key in ("q", "k", "v")] + ([tensors[n["g"]]] if self.gate else [])
        pad = -sum(r.shape[0] for r in rows) % 8        # whole groups of eight rows for the tensor-core products
        if pad:
            rows.append(torch.zeros(pad, self.width, dtype=rows[0].dtype, device=rows[0].device))
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.cols = (0, self.q_dim, self.q_dim + self.k_dim)
        self.col_g = self.q_dim + self.k_dim + self.v_dim
        self.b_qkv = torch.cat([tensors[n[k] + ".b"].float() for k in ("q", "k", "v")]).contiguous() if self.bias else None
        self.q_weight = self.k_weight = None
        if self.qk_norm:
            self.q_weight = tensors[n["q_norm"]].float()[None, :].expand(MAPS * self.heads, self.dim).contiguous()
            self.k_weight = tensors[n["k_norm"]].float().contiguous()
        l = {key: tensors[n[key]].double() for key in ("lq1", "lk1", "lq2", "lk2")}
        self.lam = float(torch.exp((l["lq1"] * l["lk1"]).sum()) - torch.exp((l["lq2"] * l["lk2"]).sum())) + self.diff
        self.w_o = tensors[n["o"]].contiguous()

    def forward(self, ctx, h, cache, residual=None):
        b, ops, ws = ctx.batch, self.ops, ctx.ws
        T = h.shape[0]
        proj = ws.get("attn_proj", (T, self.w_in.shape[0]), torch.float32)
        ops.linear(h, self.w_in, proj)
        q = ws.get("q_heads", (T, MAPS * self.heads, self.dim), self.dtype)
        ops.qk_norm_rope_append(proj, self.cols, q, cache.k, cache.v, b.positions, b.token_req, cache.block_table,
                                MAPS * self.heads, MAPS * self.kv_heads, self.dim, self.vdim, self.q_weight, self.k_weight, self.eps,
                                self.rotary, cache.page_size, bias=self.b_qkv, maps=MAPS)
        out = ws.get("attn_ctx", (T, self.ctx_dim), self.dtype)
        gate = proj[:, self.col_g:self.col_g + self.heads] if self.gate else None
        ops.differential_attention(ctx, q.view(T, self.heads, MAPS * self.dim), cache.k, cache.v, cache.block_table, out, self.scale,
                                   self.window or 0, cache.page_size, self.lam, 1.0 - self.diff, self.eps, gate)
        if residual is not None:
            ops.linear(out, self.w_o, residual, accumulate=True)
            return None
        y = ws.get("mixer_out", (T, self.width), torch.float32)
        ops.linear(out, self.w_o, y)
        return y
