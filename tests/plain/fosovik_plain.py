"""The Fosovik design, plain: numpy, 64-bit, whole sequences, no cache, one function per mechanism.

The oracle of the tests. Written from the design's equations, in the notation below; it shares no
code with ``garuda_b200``.

  squash(v)      = tanh(a v) * w + b                         (the norm: no mean, no variance)
  layer          : h = squash_1(x);  x <- x + mixer(h) + ff(h)
  logits         = W_head squash_final(x),  x_0 = E[token] * embedding_scale
"""
import math

import numpy as np


def squash(v, W, name):
    return np.tanh(float(W[name + ".alpha"]) * v) * W[name] + W[name + ".b"]


def unit_rms(v, eps):
    return v / np.sqrt(np.mean(v * v, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu_erf(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def dense_ff(W, p, limit, h):
    g = np.minimum(h @ W[p + "gate"].T, limit)
    u = np.clip(h @ W[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def routed_ff(W, p, top, h):
    """Every token's ``top`` experts by their share of the softmax over all experts; shares not renormalized."""
    z = h @ W[p + "router"].T
    s = np.exp(z - z.max(axis=-1, keepdims=True))
    s /= s.sum(axis=-1, keepdims=True)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e in np.argsort(-s[t], kind="stable")[:top]:
            out[t] += s[t, e] * (gelu_erf(h[t] @ W[f"{p}e{e}.up"].T) @ W[f"{p}e{e}.down"].T)
    return out


def softmax_sink(s, sink):
    """Rows of ``s`` (masked entries -inf) through a softmax whose denominator also holds exp(sink)."""
    m = np.maximum(s.max(axis=-1, keepdims=True), sink)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - m))


def query_factor(positions, coef, every):
    """1 + coef ln(floor((p + 1) / every) + 1)"""
    return 1.0 + coef * np.log(np.floor((np.asarray(positions, dtype=np.float64) + 1.0) / every) + 1.0)


def keys_and_values(W, p, m, eps, h):
    T, G = h.shape[0], m["kv_heads"]
    return unit_rms((h @ W[p + "k"].T).reshape(T, G, m["dim"]), eps), (h @ W[p + "v"].T).reshape(T, G, m["vdim"])


def attention(W, p, m, eps, h, kv):
    """``kv``: the keys (normed) and values that this layer reads, its own or another layer's."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    k, v = kv
    q = unit_rms((h @ W[p + "q"].T).reshape(T, H, m["dim"]), eps)
    if m.get("q_temp"):
        q = q * query_factor(np.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    causal = np.tril(np.ones((T, T), dtype=bool))
    out = np.zeros((T, H, m["vdim"]))
    for n in range(H):
        g = n // (H // G)
        s = np.where(causal, (q[:, n] @ k[:, g].T) * m["scale"], -np.inf)
        out[:, n] = softmax_sink(s, W[p + "sink"][n]) @ v[:, g]
    return out.reshape(T, -1) @ W[p + "o"].T


def causal_conv(u, taps, bias):
    """``y_t = bias + sum_j taps[:, j] u_(t - n + 1 + j)`` with ``n`` taps, zeros before the first token."""
    T, n = u.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, u.shape[1])), u], axis=0)
    return bias[None, :] + sum(padded[j:j + T] * taps[:, j][None, :] for j in range(n))


def state_space(x, B, C, dt, rate, D):
    """One head: ``S_t = exp(-rate dt_t) S_(t-1) + dt_t B_t x_t^T``, ``y_t = S_t^T C_t + D x_t``; ``x [T, P]``, ``B, C [T, N]``."""
    S = np.zeros((B.shape[1], x.shape[1]))
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = math.exp(-rate * dt[t]) * S + dt[t] * np.outer(B[t], x[t])
        y[t] = S.T @ C[t] + D * x[t]
    return y


def grouped_rms(v, groups, eps):
    T, n = v.shape
    return unit_rms(v.reshape(T, groups, n // groups), eps).reshape(T, n)


def mamba2(W, p, m, eps, h):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner, GN = H * P, G * N
    row = h @ W[p + "in"].T
    z, mixed, dt = row[:, :inner], row[:, inner:2 * inner + 2 * GN], row[:, 2 * inner + 2 * GN:]
    mixed = silu(causal_conv(mixed, W[p + "conv"], W[p + "conv.b"]))
    x = mixed[:, :inner].reshape(T, H, P)
    B = mixed[:, inner:inner + GN].reshape(T, G, N)
    C = mixed[:, inner + GN:].reshape(T, G, N)
    dt = softplus(dt + W[p + "dt_bias"])
    y = np.zeros((T, H, P))
    for n in range(H):
        g = n // (H // G)
        y[:, n] = state_space(x[:, n], B[:, g], C[:, g], dt[:, n], math.exp(W[p + "A_log"][n]), W[p + "D"][n])
    y = grouped_rms(y.reshape(T, inner) * silu(z), m["norm_groups"], eps) * W[p + "norm"]
    return y @ W[p + "o"].T


def forward(cfg, W, tokens, layers_out=None):
    """Logits ``[T, vocab]`` (64-bit) at every position. ``W``: name -> array. ``layers_out``: a list that
    receives the residual after every layer."""
    W = {n: np.asarray(a, dtype=np.float64) for n, a in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = squash(x, W, p + "norm1")
        if layer["type"] == "attention":
            source = m.get("kv_from")
            if source is None:
                kept[i] = keys_and_values(W, p + "mix.", m, eps, h)
            y = attention(W, p + "mix.", m, eps, h, kept[i if source is None else source])
        elif layer["type"] == "mamba2":
            y = mamba2(W, p + "mix.", m, eps, h)
        else:
            raise ValueError(layer["type"])
        f = layer.get("mlp")
        if f is not None:
            y = y + (dense_ff(W, p + "mlp.", f["limit"], h) if f["kind"] == "dense" else routed_ff(W, p + "mlp.", f["router"]["top"], h))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return squash(x, W, "final.norm") @ W["head"].T
