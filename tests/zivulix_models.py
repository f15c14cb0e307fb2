"""Tiny Zivulix models for tests: configurations that differ in every size and
option, and weights reshaped so that a fault shows.

Random N(0, 0.02) weights would hide most faults: the biases would swamp the
attention's queries and keys, the latent scores would be near zero and every
softmax nearly flat, and the delta rule's gates nearly constant.  `sharpen` scales
groups of tensors so that scores spread over several units (a window that is one
token off, a wrong angle or a cap that is left out shows), the gates cover their
range and the memories last for tens of tokens.
"""

from __future__ import annotations

import os
import tempfile
from typing import Dict, Tuple

import numpy as np


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim}}}


def attention(heads, kv_heads, dim, vdim, scale, softcap, rot, mask=None, v_mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
         "rot": {"base": rot[0], "dims": rot[1]}, "v_mix": v_mix}
    if len(rot) > 2:
        m["rot"]["scaling"] = {"factor": rot[2]}
    if mask is not None:
        m["mask"] = {"size": mask}
    return {"type": "attention", "mixer": m}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def model(vocab, width, eps, layers):
    return {"architecture": "Zivulix", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [dict(l, mlp=None if ff is None else {"kind": "dense", "ff": ff}) for l, ff in layers]}


# A: every mixer, with and without a feed-forward; values wider than keys, half of each head
# rotated, a window of 20, a cap that bends the scores; two values heads a query/key head
ZIV_A = model(97, 72, 1e-5, [
    (delta(4, 2, 16, 24, 4), 96),
    (attention(6, 3, 16, 24, 0.8, 5.0, (100.0, 8, 2.0), 20), None),
    (latent(3, 16, 8, 24, 40, 0.6, 1000.0), 80),
    (attention(6, 3, 16, 24, 0.5, 4.0, (100.0, 16, 3.0), 33), 48),
    (delta(3, 3, 8, 20, 2), None),
])
# B: a width that is no multiple of 8, sizes that are no multiples of 4, one tap (no filter
# state), one key head, no window, undivided frequencies, values that are not mixed
ZIV_B = model(61, 100, 1e-3, [
    (latent(5, 6, 4, 10, 18, 1.1, 50.0), None),
    (delta(2, 1, 10, 7, 1), 52),
    (attention(5, 1, 22, 12, 0.4, 6.0, (30.0, 6), None, False), 20),
    (delta(1, 1, 33, 50, 3), None),
])
# C: heads of 128 and 64 (the tcgen05 kernel, with a cap that its scores stay far below and one
# that bends them), mixed values of equal width in heads of different sizes, a window longer than
# a page, a latent row of exactly 128
ZIV_C = model(200, 256, 1e-6, [
    (attention(8, 2, 128, 128, 0.09, 40.0, (10000.0, 64, 4.0), 70), 256),
    (latent(4, 64, 16, 32, 112, 0.2, 500000.0), 128),
    (attention(8, 4, 64, 64, 0.2, 6.0, (10000.0, 32, 1.5), 64, False), None),
    (delta(4, 2, 128, 64, 4), 96),
])
# D: a latent row wider than 256, sixteen heads on it; as many query/key heads as value heads;
# values wider than 128 columns a head
ZIV_D = model(130, 128, 1e-5, [
    (latent(16, 32, 32, 48, 288, 0.25, 10000.0), 64),
    (delta(2, 2, 72, 160, 3), 64),
    (latent(2, 8, 2, 8, 30, 0.4, 7.0), None),
])
# E: the first attention layer does not mix, the second is the first that does, two more follow;
# long windows over several pages, values narrower than keys
ZIV_E = model(77, 96, 1e-5, [
    (attention(4, 2, 32, 16, 0.5, 8.0, (10000.0, 32, 2.0), 200, False), 40),
    (attention(6, 2, 48, 16, 0.4, 9.0, (1000.0, 24, 8.0), 130), None),
    (delta(6, 2, 32, 16, 2), 32),
    (attention(4, 2, 24, 16, 0.6, 7.0, (500.0, 10, 1.0), 65), 24),
    (attention(2, 2, 16, 16, 0.7, 5.0, (100.0, 16, 4.0), 1), 24),
])

ALL = {"A": ZIV_A, "B": ZIV_B, "C": ZIV_C, "D": ZIV_D, "E": ZIV_E}

# tensor-name suffix -> (factor, offset) (the longest matching suffix counts)
SHARP = (("mix.q", (15.0, 0.0)), ("mix.k", (30.0, 0.0)), ("mix.v", (15.0, 0.0)), ("mix.uk", (15.0, 0.0)),
         ("mix.dkv", (10.0, 0.0)), ("mix.uv", (10.0, 0.0)), ("mix.b", (15.0, 0.0)), ("mix.a", (15.0, 0.0)),
         ("mix.A_log", (1.0, -2.5)), ("mix.g", (15.0, 0.0)), ("mlp.gate", (15.0, 0.0)), ("mlp.up", (15.0, 0.0)),
         ("embed.norm", (5.0, 0.0)), ("norm1", (5.0, 0.0)), ("norm2", (5.0, 0.0)), ("head", (20.0, 0.0)))

_FOLDERS: Dict[Tuple[str, int, str, object], str] = {}


def sharpened(name: str, t, mild: bool):
    best, f, o = -1, 1.0, 0.0
    for suffix, (factor, offset) in SHARP:
        if name.endswith(suffix) and len(suffix) > best:
            best, f, o = len(suffix), factor, offset
    return t * (f ** 0.5 if mild else f) + o


def model_folder(name: str, seed: int = 3, dtype: str = "float32", sharp=True) -> str:
    """A model folder with the framework's random weights, sharpened; made once.
    `sharp` "mild": the square roots of the factors, for runs in bfloat16, whose
    rounding the full factors would amplify beyond what a tolerance can tell
    from a fault."""
    from reflex_b200.weights import SafetensorsFile, write_random_model, write_safetensors

    key = (name, seed, dtype, sharp)
    if key not in _FOLDERS:
        d = tempfile.mkdtemp(prefix=f"rfx_ziv_{name}_")
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
