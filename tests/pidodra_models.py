"""Tiny Pidodra models for tests: configurations that differ in every size and
option, and weights reshaped so that a fault shows.

Random N(0, 0.02) weights would hide most faults: the sublayers' results would
vanish beside the stream, the latent scores would be near zero, every softmax and
router nearly flat and the gates near one half.  `sharpen` scales groups of tensors
so that scores spread over several units (a wrong angle, a sink that is left out or
a key far away shows), the gates cover their range and the routers decide.
"""

from __future__ import annotations

import os
import tempfile
from typing import Dict, Tuple

import numpy as np


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale, "rot": {"base": base, "dims": rot_dim}}}


def attention(heads, kv_heads, dim, vdim, scale, rot, kv_from=None):
    """rot: (base, dims) or (base, dims, (factor, original, fast, slow))."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
         "rot": {"base": rot[0], "dims": rot[1]}}
    if len(rot) > 2:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2]))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def moe(ff, experts, top, scale=None, groups=None):
    r = {"experts": experts, "top": top}
    if scale is not None:
        r["scale"] = scale
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def model(vocab, width, eps, alpha, scale, layers):
    return {"architecture": "Pidodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "embedding": {"scale": scale}, "layers": [dict(l, mlp=ff) for l, ff in layers]}


YARN_A = (100.0, 8, (4.0, 64, 8.0, 1.0))
# A: every mixer, with and without a feed-forward; values wider than keys, half of each head
# rotated with scaled frequencies; a layer that uses the one before's keys and values
PID_A = model(97, 72, 1e-5, 1.5, 2.5, [
    (latent(3, 16, 8, 24, 40, 24, 0.6, 1000.0), moe(40, 12, 3, 1.5, (4, 2))),
    (attention(6, 3, 16, 24, 0.5, YARN_A), None),
    (attention(6, 3, 16, 24, 0.35, YARN_A, 1), moe(24, 6, 2)),
    (latent(5, 8, 4, 16, 24, 32, 0.8, 50.0), None),
    (attention(4, 4, 24, 24, 0.4, (500.0, 24)), moe(32, 9, 4, 0.75, (3, 2))),
])
# B: a width that is no multiple of 8, sizes that are no multiples of 4, one key head, one
# expert chosen, as many groups as experts, a stream that is not multiplied
PID_B = model(61, 100, 1e-3, 1.0, 1.0, [
    (attention(5, 1, 22, 12, 0.4, (30.0, 6, (2.5, 40, 5.0, 0.5))), moe(21, 5, 1, 0.8)),
    (latent(5, 6, 4, 10, 15, 18, 1.1, 50.0), moe(20, 7, 3, 1.25, (7, 4))),
    (attention(5, 1, 22, 12, 0.6, (30.0, 6, (2.5, 40, 5.0, 0.5)), 0), None),
    (attention(3, 3, 10, 10, 0.7, (20.0, 2)), moe(12, 4, 4, 1.0, (2, 2))),
])
# C: heads of 128 and 64 (the tcgen05 kernels), query rows that are turned where they stand
# (128 + 64), values narrower than their keys; more experts than lanes, five of them chosen
PID_C = model(200, 256, 1e-6, 2.5, 1.5, [
    (latent(4, 128, 64, 128, 96, 64, 0.07, 500000.0), moe(64, 40, 5, 0.35, (8, 3))),
    (attention(8, 2, 128, 128, 0.15, (10000.0, 128, (8.0, 256, 16.0, 1.0))), moe(48, 8, 2, 0.25, (2, 1))),
    (attention(4, 2, 64, 32, 0.2, (10000.0, 32)), None),
    (attention(8, 2, 128, 128, 0.1, (10000.0, 128, (8.0, 256, 16.0, 1.0)), 1), moe(48, 8, 2, 0.4, (4, 3))),
    (attention(4, 2, 64, 32, 0.3, (10000.0, 32), 2), None),
])
# D: latent rows wider than 256, sixteen heads on them, a query latent wider than the model;
# values wider than 128 columns a head
PID_D = model(130, 128, 1e-5, 2.25, 0.6, [
    (latent(16, 32, 32, 48, 160, 288, 0.05, 10000.0), moe(32, 16, 2, 0.9, (8, 2))),
    (latent(2, 8, 2, 8, 24, 30, 0.4, 7.0), None),
    (latent(2, 40, 24, 160, 48, 64, 0.15, 200.0), moe(40, 64, 3, 1.5, (16, 5))),
])
# E: several layers that use one layer's keys and values, with scales of their own, and a second
# such layer; attention at both ends
YARN_E = (1000.0, 32, (16.0, 128, 4.0, 0.25))
PID_E = model(77, 96, 1e-5, 3.0, 4.0, [
    (attention(4, 2, 32, 16, 0.3, YARN_E), moe(24, 8, 2, 1.5, (4, 2))),
    (latent(3, 16, 16, 16, 32, 48, 0.5, 10000.0), moe(24, 8, 2, 1.5, (4, 2))),
    (attention(4, 2, 32, 16, 0.2, YARN_E, 0), moe(24, 8, 2, 1.5, (4, 2))),
    (attention(6, 2, 24, 48, 0.4, (300.0, 10)), None),
    (attention(6, 2, 24, 48, 0.2, (300.0, 10), 3), moe(16, 4, 1)),
    (attention(4, 2, 32, 16, 0.4, YARN_E, 0), None),
])

ALL = {"A": PID_A, "B": PID_B, "C": PID_C, "D": PID_D, "E": PID_E}

# tensor-name suffix -> (factor, offset) (the longest matching suffix counts)
SHARP = (("mix.dq", (12.0, 0.0)), ("mix.uq", (10.0, 0.0)), ("mix.dkv", (10.0, 0.0)), ("mix.uk", (10.0, 0.0)),
         ("mix.uv", (10.0, 0.0)), ("mix.q", (12.0, 0.0)), ("mix.k", (12.0, 0.0)), ("mix.v", (10.0, 0.0)),
         ("mix.g", (12.0, 0.0)), ("mix.o", (10.0, 0.0)), ("mix.sink", (4.0, 1.5)), ("mlp.router", (10.0, 0.0)),
         (".gate", (10.0, 0.0)), (".up", (10.0, 0.0)), (".down", (10.0, 0.0)), ("norm1", (4.0, -3.0)),
         ("norm2", (4.0, -3.0)), (".norm", (4.0, -3.0)), ("embed", (15.0, 0.0)), ("head", (20.0, 0.0)))
# the same where runs are in bfloat16
MILD = {".down": 1.5, "mix.o": 5.0, "mix.uk": 7.0, "mix.uq": 7.0, "mix.g": 8.0}

_FOLDERS: Dict[Tuple[str, int, str, object], str] = {}


def sharpened(name: str, t, mild: bool):
    best, f, o = "", 1.0, 0.0
    for suffix, (factor, offset) in SHARP:
        if name.endswith(suffix) and len(suffix) > len(best):
            best, f, o = suffix, factor, offset
    return t * (MILD.get(best, f) if mild else f) + o


def model_folder(name: str, seed: int = 3, dtype: str = "float32", sharp=True) -> str:
    """A model folder with the framework's random weights, sharpened; made once.
    `sharp` "mild": smaller factors, for runs in bfloat16, whose rounding the full
    ones would amplify beyond what a tolerance can tell from a fault."""
    from reflex_b200.weights import SafetensorsFile, write_random_model, write_safetensors

    key = (name, seed, dtype, sharp)
    if key not in _FOLDERS:
        d = tempfile.mkdtemp(prefix=f"rfx_pid_{name}_")
        write_random_model(ALL[name], seed, d, dtype)
        if sharp:
            path = os.path.join(d, "model.safetensors")
            f = SafetensorsFile(path)
            tensors = [(k, f.tensor(k).clone()) for k in f.keys()]
            f.close()
            write_safetensors(path, [(k, sharpened(k, t.float(), sharp == "mild").to(t.dtype)) for k, t in tensors])
        _FOLDERS[key] = d
    return _FOLDERS[key]


def tokens(n: int, vocab: int, seed: int):
    rng = np.random.default_rng(seed)
    return [int(t) for t in rng.integers(0, vocab, size=n)]
