"""A plain, slow implementation of the Pidodra design, for tests.

Whole sequences, no cache, one function per mechanism, NumPy in double
precision; it shares no code with `reflex_b200`.  Linear weights are [out, in]
and applied as y = x W^T.

The design: the token embedding times a scale; layers that norm the sum of a
multiple of the stream and what a sublayer makes of it, h = norm1(a h +
mixer(h)), h = norm2(a h + ff(h)); the mixer is a latent attention (queries
through a normed latent, keys and values from a cached normed latent, one rotated
key part all heads share, a sink in the softmax, a gate per element) or a grouped
attention (normed queries and keys, a YaRN-scaled rotation, a gate per head), which
may read the keys and values of an earlier layer; the feed-forward is a mixture of
experts chosen among the best groups, or absent; a final norm and an untied head.
"""

from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional

import numpy as np

F = np.float64


def read_safetensors(path: str) -> Dict[str, np.ndarray]:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n).decode("utf-8"))
        blob = f.read()
    out = {}
    for name, ent in header.items():
        if name == "__metadata__":
            continue
        b, e = ent["data_offsets"]
        raw = blob[b:e]
        if ent["dtype"] == "BF16":
            arr = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32)
        elif ent["dtype"] == "F32":
            arr = np.frombuffer(raw, dtype="<f4")
        elif ent["dtype"] == "I32":
            arr = np.frombuffer(raw, dtype="<i4")
        else:
            raise ValueError(f"plain reader: dtype {ent['dtype']} of {name}")
        out[name] = arr.astype(F).reshape(ent["shape"])
    return out


def read_model(model_dir: str):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))


# ------------------------------------------------------------------ elements
def rms_norm(x: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def inverse_frequencies(dims: int, base: float) -> List[float]:
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_frequencies(dims: int, base: float, factor: float, original: float, fast: float, slow: float) -> List[float]:
    """Pairs that turn more than `fast` times within `original` positions keep their
    frequency, those that turn less than `slow` times have it divided by `factor`,
    and the ones between go over linearly in the pair's index."""
    def index_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    a = max(math.floor(index_of(fast)), 0)
    b = min(math.ceil(index_of(slow)), dims - 1)
    out = []
    for i, g in enumerate(inverse_frequencies(dims, base)):
        slower = min(max((i - a) / max(b - a, 0.001), 0.0), 1.0)  # the share of the divided frequency
        out.append((g / factor) * slower + g * (1.0 - slower))
    return out


def yarn_magnitude(factor: float) -> float:
    return 0.1 * math.log(factor) + 1.0


def turn_pairs(t: np.ndarray, positions: np.ndarray, freqs, first, second, magnitude: float = 1.0) -> np.ndarray:
    """t [T, heads, n]: elements first[i] and second[i] form pair i, which turns by
    position * freqs[i]; all other elements stay."""
    if len(freqs) == 0:
        return t
    ang = positions[:, None].astype(F) * np.asarray(freqs, dtype=F)[None, :]
    c, s = np.cos(ang)[:, None, :] * magnitude, np.sin(ang)[:, None, :] * magnitude
    u, v = t[..., first], t[..., second]
    out = t.copy()
    out[..., first] = u * c - v * s
    out[..., second] = v * c + u * s
    return out


def rotate_halves(t, positions, freqs, magnitude: float = 1.0):
    half = len(freqs)
    return turn_pairs(t, positions, freqs, np.arange(half), np.arange(half) + half, magnitude)


def rotate_neighbours(t, positions, freqs, magnitude: float = 1.0):
    half = len(freqs)
    return turn_pairs(t, positions, freqs, 2 * np.arange(half), 2 * np.arange(half) + 1, magnitude)


def causal(T: int) -> np.ndarray:
    return np.arange(T)[None, :] <= np.arange(T)[:, None]


def softmax_rows(s: np.ndarray, ok: np.ndarray, sink: Optional[float] = None) -> np.ndarray:
    """Softmax over the visible scores; exp(sink), when given, joins the denominator."""
    s = np.where(ok, s, -np.inf)
    top = s.max(axis=-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.exp(s - top)
    total = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        total = total + np.exp(sink - top)
    return e / total


# ---------------------------------------------------------- latent attention
def latent_attention(h: np.ndarray, w: Dict[str, np.ndarray], m: dict, eps: float) -> np.ndarray:
    T = h.shape[0]
    H, d, r, dv, kr = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    pos = np.arange(T)
    freqs = inverse_frequencies(r, float(m["rot"]["base"]))
    cq = rms_norm(h @ w["dq"].T, w["dq.norm"], eps)
    q = (cq @ w["uq"].T).reshape(T, H, d + r)
    q_rot = rotate_neighbours(q[..., d:], pos, freqs)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :kr], w["dkv.norm"], eps)
    k_rot = rotate_neighbours(down[:, None, kr:], pos, freqs)[:, 0]
    k = (c @ w["uk"].T).reshape(T, H, d)
    v = (c @ w["uv"].T).reshape(T, H, dv)
    ok = causal(T)
    out = np.zeros((T, H, dv), dtype=F)
    for hh in range(H):
        s = (q[:, hh, :d] @ k[:, hh].T + q_rot[:, hh] @ k_rot.T) * float(m["scale"])
        out[:, hh] = softmax_rows(s, ok, float(w["sink"][hh])) @ v[:, hh]
    return (out.reshape(T, H * dv) * sigmoid(h @ w["g"].T)) @ w["o"].T


# ----------------------------------------------------------------- attention
def attention_frequencies(rot: dict):
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    if not sc:
        return inverse_frequencies(dims, base), 1.0
    return (yarn_frequencies(dims, base, float(sc["factor"]), float(sc["original"]), float(sc["fast"]),
                             float(sc["slow"])), yarn_magnitude(float(sc["factor"])))


def keys_and_values(h: np.ndarray, w: Dict[str, np.ndarray], m: dict, eps: float):
    """A layer's keys, normed and rotated, and its values: what its cache holds."""
    T = h.shape[0]
    G, d, dv = (int(m[k]) for k in ("kv_heads", "dim", "vdim"))
    freqs, mag = attention_frequencies(m["rot"])
    k = rms_norm((h @ w["k"].T).reshape(T, G, d), w["k.norm"], eps)
    return rotate_halves(k, np.arange(T), freqs, mag), (h @ w["v"].T).reshape(T, G, dv)


def attention(h: np.ndarray, w: Dict[str, np.ndarray], m: dict, eps: float, k: np.ndarray, v: np.ndarray) -> np.ndarray:
    T = h.shape[0]
    H, G, d, dv = (int(m[k_]) for k_ in ("heads", "kv_heads", "dim", "vdim"))
    freqs, mag = attention_frequencies(m["rot"])
    q = rms_norm((h @ w["q"].T).reshape(T, H, d), w["q.norm"], eps)
    q = rotate_halves(q, np.arange(T), freqs, mag)
    ok = causal(T)
    gate = sigmoid(h @ w["g"].T)  # [T, H]
    out = np.zeros((T, H, dv), dtype=F)
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * float(m["scale"])
        out[:, hh] = (softmax_rows(s, ok) @ v[:, g]) * gate[:, hh:hh + 1]
    return out.reshape(T, H * dv) @ w["o"].T


# --------------------------------------------------------- mixture of experts
def choose_experts(scores: np.ndarray, top: int, groups: Optional[dict]) -> List[int]:
    """The `top` experts of largest score among the groups of largest best score;
    ties go to the lower index."""
    E = len(scores)
    allowed = np.ones(E, dtype=bool)
    if groups:
        count, keep = int(groups["count"]), int(groups["keep"])
        best = scores.reshape(count, E // count).max(axis=1)
        kept = sorted(range(count), key=lambda g: (-best[g], g))[:keep]
        allowed = np.repeat([g in kept for g in range(count)], E // count)
    order = sorted((e for e in range(E) if allowed[e]), key=lambda e: (-scores[e], e))
    return order[:top]


def expert(h: np.ndarray, w: Dict[str, np.ndarray], e: int) -> np.ndarray:
    return (silu(h @ w[f"e{e}.gate"].T) * (h @ w[f"e{e}.up"].T)) @ w[f"e{e}.down"].T


def experts_ff(h: np.ndarray, w: Dict[str, np.ndarray], mlp: dict) -> np.ndarray:
    r = mlp["router"]
    z = h @ w["router"].T
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s = s / s.sum(axis=1, keepdims=True)
    factor = float(r.get("scale", 1.0))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose_experts(s[t], int(r["top"]), r.get("groups")):
            out[t] += s[t, e] * factor * expert(h[t], w, e)
    return out


# ------------------------------------------------------------------ the model
def sub(tensors: Dict[str, np.ndarray], prefix: str) -> Dict[str, np.ndarray]:
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def layer_forward(x, cfg, tensors, li, kept):
    """`kept`: layer index -> (keys, values) of the attention layers run so far."""
    L = cfg["layers"][li]
    eps, alpha = float(cfg["norm"]["eps"]), float(cfg["postln_alpha"])
    pre = f"l{li}."
    w, m = sub(tensors, pre + "mix."), L["mixer"]
    if L["type"] == "latent_attention":
        y = latent_attention(x, w, m, eps)
    elif L["type"] == "attention":
        source = m.get("kv_from")
        if source is None:
            kept[li] = keys_and_values(x, w, m, eps)
            source = li
        y = attention(x, w, m, eps, *kept[int(source)])
    else:
        raise ValueError(L["type"])
    x = rms_norm(alpha * x + y, tensors[pre + "norm1"], eps)
    if L.get("mlp") is not None:
        x = rms_norm(alpha * x + experts_ff(x, sub(tensors, pre + "mlp."), L["mlp"]), tensors[pre + "norm2"], eps)
    return x


def forward(cfg, tensors, tokens, want=None, layers_out: Optional[list] = None) -> np.ndarray:
    """Logits [len(want) or T, vocab] of one whole sequence."""
    x = tensors["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
    kept: dict = {}
    for li in range(len(cfg["layers"])):
        x = layer_forward(x, cfg, tensors, li, kept)
        if layers_out is not None:
            layers_out.append(x.copy())
    x = rms_norm(x, tensors["final.norm"], float(cfg["norm"]["eps"]))
    if want is not None:
        x = x[np.asarray(want, dtype=np.int64)]
    return x @ tensors["head"].T
