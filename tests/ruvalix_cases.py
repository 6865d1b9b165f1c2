"""Tiny Ruvalix configurations for the tests, their model folders and the plain model's logits.

The configurations differ from one another in every size and option: one, two and three query heads per
key head; maps and values that are unequal, odd and no multiple of 8; a rotation of a part of a map's channels, of
all of them, stretched, not stretched and none; windows of 7 to 100 positions, two in one model, and none;
memories with one to three heads, wider keys than values and the reverse, sizes that the tensor-core kernel takes and
ones it does not; experts with and without identity ones, in one to four groups of which one or more are
kept, all chosen, one chosen; with and without a shared expert; layers without a feed-forward; no loop, loops from the
first layer, over the last, of one layer, and one, two and three passes.
"""
import tempfile

import numpy as np
import torch


def _att(heads, kv_heads, dim, vdim, scale, diff, window=None, rot=None, stretch=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if window:
        m["mask"] = {"size": window}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if stretch:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), stretch))
    return m


def _mem(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def _moe(experts, top, ff, identity=0, groups=None, shared=None):
    r = {"experts": experts, "top": top}
    if identity:
        r["identity"] = identity
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    f = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# sizes no tensor-core kernel takes (width 44, maps of 10, values of 13, memories of 7 x 11); the last two layers looped
RA = {"architecture": "Ruvalix", "vocab": 96, "width": 44, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 2},
      "layers": [_layer("mlstm", _mem(3, 7, 11, 6.0), _moe(5, 3, 24, identity=1, groups=(3, 2), shared=20)),
                 _layer("attention", _att(6, 2, 10, 13, 0.4, 0.3, window=7, rot=(100.0, 6), stretch=(3.0, 60, 4.0, 0.5)), _moe(4, 4, 18, shared=30)),
                 _layer("mlstm", _mem(2, 12, 5, 15.0), None)]}

# sizes the tensor-core kernels take (maps of 32, values of 64, memories of 64 x 32); a loop of three passes
RB = {"architecture": "Ruvalix", "vocab": 160, "width": 128, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 2, "times": 3},
      "layers": [_layer("attention", _att(4, 2, 32, 64, 0.2, 0.7, window=40, rot=(10000.0, 32), stretch=(4.0, 128, 16.0, 1.0)),
                        _moe(6, 2, 64, identity=2, groups=(4, 2), shared=96)),
                 _layer("mlstm", _mem(2, 64, 32, 10.0), _moe(8, 3, 64)),
                 _layer("attention", _att(2, 2, 16, 16, 0.4, 0.2, window=100), _moe(3, 1, 128, identity=1, groups=(2, 1), shared=64)),
                 _layer("mlstm", _mem(1, 16, 48, 15.0), _moe(6, 4, 40, identity=6, groups=(3, 2)))]}

# one layer of attention over every earlier position and nothing else; rotated, not stretched
RC = {"architecture": "Ruvalix", "vocab": 64, "width": 32, "norm": {"eps": 1e-5},
      "layers": [_layer("attention", _att(2, 1, 15, 15, 0.6, 0.5, rot=(1000.0, 14)), None)]}

# wide heads; a loop of one pass over the last layer
RD = {"architecture": "Ruvalix", "vocab": 200, "width": 72, "norm": {"eps": 1e-5}, "loop": {"start": 2, "stop": 3, "times": 1},
      "layers": [_layer("mlstm", _mem(2, 128, 64, 15.0), _moe(7, 2, 40, shared=72)),
                 _layer("attention", _att(3, 1, 64, 128, 0.25, 0.8, window=33, rot=(500000.0, 24), stretch=(8.0, 4096, 32.0, 1.0)), None),
                 _layer("attention", _att(2, 2, 48, 80, 0.3, 0.6, window=64, rot=(10000.0, 48)), _moe(2, 1, 72, identity=2, shared=40))]}

CASES = {"RA": (RA, 61), "RB": (RB, 62), "RC": (RC, 63), "RD": (RD, 64)}

# Random N(0, 0.02) weights leave every expert alike, every memory small and the logits flat; these factors spread the
# router's logits, the memories' inputs and the logits, and keep some memories for hundreds of tokens. (The attention's scores are spread by the configurations' scale,
# since queries and keys are normed; a factor matches every tensor whose name holds the key.)
SHARPEN = {"mix.q": 6.0, "mix.k": 6.0, "mix.v": 6.0, "mix.i": 3.0, "mix.f.b": 2.0, "mix.o": 5.0, "mix.g": 4.0, ".router": 4.0, ".gate": 5.0, ".up": 5.0,
           ".down": 5.0, "loop.in": 8.0, "head": 4.0}
# (the factor on mix.q and mix.k must not reach the norms' weights)
UNSCALED = ("q.norm", "k.norm")

_DIRS, _PLAIN = {}, {}


def write(folder, cfg, seed, store_dtype):
    """A model folder with sharpened random weights."""
    from garuda_b200.weights import SafetensorsFolder, write_random_model, write_safetensors
    d = write_random_model(folder, cfg, seed, store_dtype=store_dtype, scale=SHARPEN)
    f = SafetensorsFolder(d)
    t = {n: f.tensor(n).clone() for n in f.names()}
    for n in t:
        if n.endswith(UNSCALED):
            t[n] = (t[n].float() / 6.0).to(store_dtype)
    write_safetensors(d + "/model.safetensors", t)
    return d


def model_dir(name: str, store_dtype=torch.float32) -> str:
    key = (name, store_dtype)
    if key not in _DIRS:
        cfg, seed = CASES[name]
        _DIRS[key] = write(tempfile.mkdtemp(prefix=f"garuda_ruvalix_{name}_"), cfg, seed, store_dtype)
    return _DIRS[key]


def weights(name: str, store_dtype=torch.float32) -> dict:
    from tests.helpers import folder_weights
    return folder_weights(model_dir(name, store_dtype))


def plain_logits(name: str, store_dtype, tokens) -> np.ndarray:
    from tests.plain import ruvalix_plain
    key = (name, store_dtype, tuple(tokens))
    if key not in _PLAIN:
        _PLAIN[key] = ruvalix_plain.forward(CASES[name][0], weights(name, store_dtype), tokens).astype(np.float32)
    return _PLAIN[key]


def random_tokens(name: str, n: int, seed: int):
    return np.random.default_rng(seed).integers(0, CASES[name][0]["vocab"], n).tolist()


def edge_model(folder, store_dtype, window=40, vocab=80):
    """One attention layer whose query of token 1 finds the key of token 0 through a channel that is not rotated, in the
    first map alone, wherever both are. Returns (folder, configuration)."""
    from garuda_b200.weights import SafetensorsFolder, write_safetensors
    cfg = {"architecture": "Ruvalix", "vocab": vocab, "width": 48, "norm": {"eps": 1e-6},
           "layers": [_layer("attention", _att(2, 1, 16, 32, 1.0, 0.4, window=window, rot=(10000.0, 8), stretch=(2.0, 100, 8.0, 1.0)),
                             _moe(3, 2, 16, identity=1, shared=16))]}
    d = write(folder, cfg, 3, store_dtype)
    f = SafetensorsFolder(d)
    t = {n: f.tensor(n).clone() for n in f.names()}
    t["embed"][:, :2] = 0.0
    t["embed"][0], t["embed"][1] = 0.0, 0.0
    t["embed"][0, 0], t["embed"][1, 1] = 1.0, 1.0
    for name, heads, channel in (("q", 2, 1), ("k", 1, 0)):
        w = t[f"l0.mix.{name}"].view(heads, 2, 16, 48)
        w[..., :2] = 0.0
        w[:, 0, 15] = 0.0
        w[:, 0, 15, channel] = 40.0
        t[f"l0.mix.{name}.b"].view(heads, 2, 16)[:, 0, 15] = 0.0
    write_safetensors(d + "/model.safetensors", t)
    return d, cfg
