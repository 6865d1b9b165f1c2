"""Tiny Fosovik configurations for the tests, their model folders and the plain model's logits.

The configurations differ from one another in every size and option: one, two and three query heads per
key head; key and value widths that are unequal, odd and no multiple of 8; queries that grow every 5, 16
and 37 positions, by a negative factor, and not at all; a layer that reads another's keys and values
right behind it, two that read the same one, and none; recurrences with 1 to 5 taps, one to three
groups, states narrower and wider than the heads, one to six parts in the norm; state and head widths
that the tensor-core kernel takes and ones it does not; layers without a feed-forward; one expert of
several, all of them, and more.
"""
import tempfile

import numpy as np
import torch


def _att(heads, kv_heads, dim, vdim, scale, temp=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _ssm(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# both mixers, both feed-forwards; sizes no tensor-core kernel takes (width 44, heads of 12, 20, 9, a state of 10)
FA = {"architecture": "Fosovik", "vocab": 96, "width": 44, "embedding": {"scale": 3.0}, "norm": {"eps": 1e-5},
      "layers": [_layer("mamba2", _ssm(6, 9, 10, 3, 3, 6), _moe(5, 2, 24)),
                 _layer("attention", _att(4, 2, 12, 20, 0.7, temp=(0.4, 5)), _dense(56, 0.9)),
                 _layer("attention", _att(6, 2, 12, 20, 0.5, temp=(-0.1, 16), kv_from=1), _moe(4, 4, 18)),
                 _layer("mamba2", _ssm(2, 20, 7, 1, 1, 1), None),
                 _layer("mamba2", _ssm(5, 4, 33, 5, 5, 2), _dense(40, 2.0))]}

# sizes the tensor-core kernels take (heads of 64 and 32, states of 64, 16 and 128); two layers read the keys of one
FB = {"architecture": "Fosovik", "vocab": 160, "width": 128, "embedding": {"scale": 9.0}, "norm": {"eps": 1e-6},
      "layers": [_layer("attention", _att(4, 2, 64, 32, 0.6, temp=(0.3, 37)), _moe(8, 3, 64)),
                 _layer("mamba2", _ssm(8, 32, 64, 2, 4, 2), _moe(6, 1, 128)),
                 _layer("attention", _att(2, 2, 64, 32, 0.5, kv_from=0), _dense(192, 1.2)),
                 _layer("mamba2", _ssm(4, 64, 16, 1, 2, 4), None),
                 _layer("attention", _att(6, 2, 64, 32, 0.4, temp=(0.7, 64), kv_from=0), None),
                 _layer("mamba2", _ssm(2, 16, 128, 2, 3, 1), _dense(256, 3.0))]}

# one layer of attention and nothing else
FC = {"architecture": "Fosovik", "vocab": 64, "width": 32, "embedding": {"scale": 2.0}, "norm": {"eps": 1e-5},
      "layers": [_layer("attention", _att(2, 1, 15, 15, 1.2, temp=(0.5, 9)), None)]}

# recurrences with wide states between an attention and another that reads it from far behind
FD = {"architecture": "Fosovik", "vocab": 200, "width": 72, "embedding": {"scale": 5.5}, "norm": {"eps": 1e-5},
      "layers": [_layer("attention", _att(3, 1, 24, 48, 0.5, temp=(1.5, 100)), _moe(7, 3, 40)),
                 _layer("mamba2", _ssm(3, 48, 80, 1, 4, 3), _dense(144, 0.5)),
                 _layer("mamba2", _ssm(4, 16, 256, 4, 4, 1), _moe(2, 1, 72)),
                 _layer("attention", _att(1, 1, 24, 48, 0.9, kv_from=0), _dense(80, 1.0))]}

CASES = {"FA": (FA, 51), "FB": (FB, 52), "FC": (FC, 53), "FD": (FD, 54)}

# Random N(0, 0.02) weights leave every expert alike, every state small and the logits flat; these factors
# spread the router's logits, the recurrences' inputs and the logits. (The attention's scores are spread by the
# configurations' scale, since queries and keys are normed; a factor matches every tensor whose name holds the key.)
SHARPEN = {"mix.in": 6.0, "mix.v": 6.0, "mix.o": 5.0, ".router": 12.0, ".gate": 5.0, ".up": 5.0, ".down": 5.0, "embed": 20.0,
           "head": 4.0}

_DIRS, _PLAIN = {}, {}


def model_dir(name: str, store_dtype=torch.float32) -> str:
    from garuda_b200.weights import write_random_model
    key = (name, store_dtype)
    if key not in _DIRS:
        cfg, seed = CASES[name]
        d = tempfile.mkdtemp(prefix=f"garuda_fosovik_{name}_")
        write_random_model(d, cfg, seed, store_dtype=store_dtype, scale=SHARPEN)
        _DIRS[key] = d
    return _DIRS[key]


def weights(name: str, store_dtype=torch.float32) -> dict:
    from tests.helpers import folder_weights
    return folder_weights(model_dir(name, store_dtype))


def plain_logits(name: str, store_dtype, tokens) -> np.ndarray:
    from tests.plain import fosovik_plain
    key = (name, store_dtype, tuple(tokens))
    if key not in _PLAIN:
        _PLAIN[key] = fosovik_plain.forward(CASES[name][0], weights(name, store_dtype), tokens).astype(np.float32)
    return _PLAIN[key]


def random_tokens(name: str, n: int, seed: int):
    return np.random.default_rng(seed).integers(0, CASES[name][0]["vocab"], n).tolist()
