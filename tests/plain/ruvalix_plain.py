"""The Ruvalix design, plain: numpy, 64-bit, whole sequences, no cache, one function per mechanism.

The oracle of the tests. Written from the design's equations, in the notation below; it shares no
code with ``garuda_b200``.

  N_w(v)     = v / sqrt(mean(v^2) + eps) * (1 + w)
  x_0        = N_embed(E[token])
  a pass t   : x <- W_in [x ; x_0] + step_t, then the looped layers
  layer      : x <- x + N_1b(mixer(N_1(x)));  x <- x + N_2b(ff(N_2(x)))
  logits     = W_head N_final(x)
"""
import math

import numpy as np


def unit_rms(v, eps):
    return v / np.sqrt(np.mean(v * v, axis=-1, keepdims=True) + eps)


def offset_norm(v, w, eps):
    return unit_rms(v, eps) * (1.0 + w)


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


# ------------------------------------------------------------------ matrix memory
def matrix_memory(q, k, v, log_in, log_forget):
    """One head. ``q, k [T, D]`` (``q`` already scaled), ``v [T, P]``; gates as logarithms ``[T]``. The memory and its
    normalizer are kept divided by ``exp(m)``, ``m`` a running maximum that starts at zero."""
    S, n, m = np.zeros((k.shape[1], v.shape[1])), np.zeros(k.shape[1]), 0.0
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        before = log_forget[t] + m
        m = max(before, log_in[t])
        keep, put = math.exp(before - m), math.exp(log_in[t] - m)
        S = keep * S + put * np.outer(k[t], v[t])
        n = keep * n + put * k[t]
        out[t] = (q[t] @ S) / (max(abs(float(n @ q[t])), math.exp(-m)) + 1e-6)
    return out


def mlstm(W, p, c, eps, h):
    T, H, D, P = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q = (h @ W[p + "q"].T).reshape(T, H, D) / math.sqrt(D)
    k = (h @ W[p + "k"].T).reshape(T, H, D)
    v = (h @ W[p + "v"].T).reshape(T, H, P)
    log_in = soft_cap(h @ W[p + "i"].T + W[p + "i.b"], c["gate_cap"])
    log_forget = log_sigmoid(soft_cap(h @ W[p + "f"].T + W[p + "f.b"], c["gate_cap"]))
    o = np.stack([matrix_memory(q[:, n], k[:, n], v[:, n], log_in[:, n], log_forget[:, n]) for n in range(H)], axis=1)
    o = unit_rms(o, eps).reshape(T, H * P) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


# ------------------------------------------------------------------ differential attention
def yarn(base, dims, scaling):
    """Frequencies ``[dims / 2]`` and the factor on cosines and sines."""
    freq = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return freq, 1.0
    factor = float(scaling["factor"])

    def turns(t):         # the (fractional) channel whose wave makes t turns over the original length
        return dims * math.log(scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(turns(scaling["fast"])), 0), min(math.ceil(turns(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return freq / factor * ramp + freq * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_half(x, positions, freq, factor):
    """``x [T, H, D]``: channel i with channel i + dims / 2 of the first ``dims = 2 len(freq)`` channels."""
    n = len(freq)
    a = np.asarray(positions, dtype=np.float64)[:, None, None] * freq
    c, s = np.cos(a) * factor, np.sin(a) * factor
    u, v = x[..., :n], x[..., n:2 * n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * n:]], axis=-1)


def softmax(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def window_mask(T, size):
    """Query i (a row) sees key j: 0 <= i - j < size."""
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (back >= 0) & (back < (size if size else T + 1))


def mixing_number(W, p, diff):
    return math.exp(float(np.sum(W[p + "lq1"] * W[p + "lk1"]))) - math.exp(float(np.sum(W[p + "lq2"] * W[p + "lk2"]))) + diff


def difference_of_maps(a1, a2, lam, diff, eps):
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention(W, p, c, eps, h):
    T, H, G, D, P = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = (h @ W[p + "q"].T + W[p + "q.b"]).reshape(T, 2 * H, D)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).reshape(T, 2 * G, D)
    v = (h @ W[p + "v"].T + W[p + "v.b"]).reshape(T, G, P)
    q, k = unit_rms(q, eps) * W[p + "q.norm"], unit_rms(k, eps) * W[p + "k.norm"]
    rot = c.get("rot")
    if rot:
        freq, factor = yarn(rot["base"], rot["dims"], rot.get("scaling"))
        q, k = (rotate_half(x, np.arange(T), freq, factor) for x in (q, k))
    mask = window_mask(T, (c.get("mask") or {}).get("size"))
    lam = mixing_number(W, p, c["diff"])
    gates = sigmoid(h @ W[p + "g"].T)
    out = np.zeros((T, H, P))
    for n in range(H):
        g = n // (H // G)
        maps = [softmax(np.where(mask, (q[:, 2 * n + j] @ k[:, 2 * g + j].T) * c["scale"], -np.inf)) @ v[:, g] for j in (0, 1)]
        out[:, n] = difference_of_maps(maps[0], maps[1], lam, c["diff"], eps) * gates[:, n:n + 1]
    return out.reshape(T, H * P) @ W[p + "o"].T


# ------------------------------------------------------------------ feed-forward
def gated_ff(W, p, h):
    g = h @ W[p + "gate"].T
    return (g * sigmoid(g) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def choose(s, correction, top, count, keep):
    """The chosen experts of one token: the largest of ``s + correction`` among the ``keep`` best of ``count`` groups."""
    c = s + correction
    size = len(c) // count
    best = [c[g * size:(g + 1) * size].max() for g in range(count)]
    allowed = np.full(len(c), -np.inf)
    for g in np.argsort(-np.array(best), kind="stable")[:keep]:
        allowed[g * size:(g + 1) * size] = c[g * size:(g + 1) * size]
    return np.argsort(-allowed, kind="stable")[:top]


def routed_ff(W, p, f, h):
    r = f["router"]
    E = r["experts"]
    s = softmax(h @ W[p + "router"].T)
    groups = r.get("groups") or {"count": 1, "keep": 1}
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose(s[t], W[p + "correction"], r["top"], groups["count"], groups["keep"]):
            out[t] += s[t, e] * (gated_ff(W, f"{p}e{e}.", h[t]) if e < E else h[t])
    if f.get("shared"):
        out = out + gated_ff(W, p + "shared.", h)
    return out


# ------------------------------------------------------------------ the model
def run_order(cfg):
    """(layer, pass or None) in the order of the runs; the pass is given with the first layer of each."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, W, tokens, layers_out=None):
    """Logits ``[T, vocab]`` (64-bit) at every position. ``W``: name -> array. ``layers_out``: a list that
    receives the residual after every layer run."""
    W = {n: np.asarray(a, dtype=np.float64) for n, a in W.items()}
    eps = cfg["norm"]["eps"]
    x0 = offset_norm(W["embed"][np.asarray(tokens)], W["embed.norm"], eps)
    x = x0
    for i, t in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = np.concatenate([x, x0], axis=-1) @ W["loop.in"].T + W["loop.step"][t]
        mixer = {"attention": attention, "mlstm": mlstm}[layer["type"]]
        h = offset_norm(x, W[p + "norm1"], eps)
        x = x + offset_norm(mixer(W, p + "mix.", layer["mixer"], eps, h), W[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            h = offset_norm(x, W[p + "norm2"], eps)
            x = x + offset_norm(routed_ff(W, p + "mlp.", layer["mlp"], h), W[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return offset_norm(x, W["final.norm"], eps) @ W["head"].T
