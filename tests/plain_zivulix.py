"""A plain, slow implementation of the Zivulix design, for tests.

Whole sequences, no cache, one function per mechanism, NumPy in double
precision; it shares no code with `reflex_b200`.  Linear weights are [out, in]
and applied as y = x W^T.

The design: the normed token embedding; layers x <- x + norm1(mixer(x)),
x <- x + norm2(ff(x)) (the sublayers read x itself; norm weights are stored
around zero, applied as 1 + w); the mixer is a latent attention (keys and values
from a cached low-rank latent, beside it one rotated key part that all heads
share), a grouped attention (biases, a rotation with divided frequencies, unit
root-mean-square queries and keys after it, capped scores, a sliding window,
values mixed with the first such layer's) or a gated delta rule (short filters,
unit keys and queries, a decay and a write rate per head, a gated per-head
norm); the feed-forward is a gated one with the tanh form of gelu, or absent;
a final norm and an untied head.
"""

from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, Optional

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
def rms_unit(x: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def norm_around_zero(x: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    return rms_unit(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(t: np.ndarray, positions: np.ndarray, dims: int, base: float, divide: float = 1.0) -> np.ndarray:
    """t [T, heads, n]: among the first `dims` dimensions i pairs with i + dims / 2 and
    the pair turns by position * base^(-2i / dims) / divide."""
    half = dims // 2
    if half == 0:
        return t
    freqs = np.array([base ** (-2.0 * i / dims) / divide for i in range(half)], dtype=F)
    ang = positions[:, None].astype(F) * freqs[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    out = t.copy()
    u, v = t[..., :half], t[..., half:2 * half]
    out[..., :half] = u * c - v * s
    out[..., half:2 * half] = v * c + u * s
    return out


def visible(T: int, window: Optional[int]) -> np.ndarray:
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    ok = j <= i
    if window:
        ok &= (i - j) < window
    return ok


def softmax_rows(s: np.ndarray, ok: np.ndarray) -> np.ndarray:
    s = np.where(ok, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


# ---------------------------------------------------------- latent attention
def latent_attention(h: np.ndarray, w: Dict[str, np.ndarray], m: dict, eps: float) -> np.ndarray:
    """Per head a key [W_uk c | rotated part shared by all heads] and a value W_uv c."""
    T = h.shape[0]
    H, d, r, dv, kr = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    pos = np.arange(T)
    base = float(m["rot"]["base"])
    q = (h @ w["q"].T).reshape(T, H, d + r)
    q_rot = rotate(q[..., d:], pos, r, base)
    down = h @ w["dkv"].T
    c = rms_unit(down[:, :kr], eps) * w["dkv.norm"]
    k_rot = rotate(down[:, None, kr:], pos, r, base)[:, 0]
    k = (c @ w["uk"].T).reshape(T, H, d)
    v = (c @ w["uv"].T).reshape(T, H, dv)
    ok = visible(T, None)
    out = np.zeros((T, H, dv), dtype=F)
    for hh in range(H):
        s = (q[:, hh, :d] @ k[:, hh].T + q_rot[:, hh] @ k_rot.T) * float(m["scale"])
        out[:, hh] = softmax_rows(s, ok) @ v[:, hh]
    return out.reshape(T, H * dv) @ w["o"].T


# ----------------------------------------------------------------- attention
def mixed_values(v: np.ndarray, m: dict, w: Dict[str, np.ndarray], carry: dict) -> np.ndarray:
    """Values of a layer that mixes: the first such layer's stay and are remembered,
    a later one's become (1 - lambda) v + lambda v_first."""
    if not m.get("v_mix"):
        return v
    if "v_first" not in carry:
        carry["v_first"] = v
        return v
    lam = float(np.asarray(w["vmix"]).reshape(()))
    return (1.0 - lam) * v + lam * carry["v_first"]


def attention(h: np.ndarray, w: Dict[str, np.ndarray], m: dict, eps: float, carry: dict) -> np.ndarray:
    T = h.shape[0]
    H, G, d, dv = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    q = (h @ w["q"].T + w["q.b"]).reshape(T, H, d)
    k = (h @ w["k"].T + w["k.b"]).reshape(T, G, d)
    v = (h @ w["v"].T + w["v.b"]).reshape(T, G, dv)
    rot = m["rot"]
    divide = float(rot["scaling"]["factor"]) if rot.get("scaling") else 1.0
    pos = np.arange(T)
    q = rms_unit(rotate(q, pos, int(rot["dims"]), float(rot["base"]), divide), eps)
    k = rms_unit(rotate(k, pos, int(rot["dims"]), float(rot["base"]), divide), eps)
    v = mixed_values(v, m, w, carry)
    ok = visible(T, int(m["mask"]["size"]) if m.get("mask") else None)
    cap = float(m["softcap"])
    out = np.zeros((T, H, dv), dtype=F)
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * float(m["scale"])
        out[:, hh] = softmax_rows(cap * np.tanh(s / cap), ok) @ v[:, g]
    return out.reshape(T, H * dv) @ w["o"].T


# ----------------------------------------------------------- gated delta rule
UNIT_EPS = 1e-6   # under the root of the unit keys and queries


def causal_conv(x: np.ndarray, taps_w: np.ndarray) -> np.ndarray:
    """x [T, C]; taps_w [C, taps], the last tap meets the current token; zeros before the start."""
    T, C = x.shape
    taps = taps_w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, C), dtype=F), x])
    out = np.zeros((T, C), dtype=F)
    for j in range(taps):
        out += padded[j:j + T] * taps_w[:, j]
    return out


def unit(x: np.ndarray) -> np.ndarray:
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + UNIT_EPS)


def gated_delta_scan(q, k, v, decay, beta):
    """q, k [T, G, d], v [T, H, dv], decay, beta [T, H]; head h reads q/k head
    h // (H / G).  S <- decay S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    T, H, dv = v.shape
    G, d = q.shape[1:]
    o = np.zeros_like(v)
    S = np.zeros((H, d, dv), dtype=F)
    for t in range(T):
        for hh in range(H):
            g = hh // (H // G)
            S[hh] = decay[t, hh] * S[hh]
            u = beta[t, hh] * (v[t, hh] - S[hh].T @ k[t, g])
            S[hh] += np.outer(k[t, g], u)
            o[t, hh] = S[hh].T @ q[t, g]
    return o


def delta_mixer(h: np.ndarray, w: Dict[str, np.ndarray], m: dict, eps: float) -> np.ndarray:
    T = h.shape[0]
    H, G, d, dv = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.reshape(T, G, d)) * d ** -0.5
    k = unit(k.reshape(T, G, d))
    beta = sigmoid(h @ w["b"].T)
    decay = np.exp(-np.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o = gated_delta_scan(q, k, v.reshape(T, H, dv), decay, beta)
    o = rms_unit(o, eps) * w["norm"] * silu(h @ w["g"].T).reshape(T, H, dv)
    return o.reshape(T, H * dv) @ w["o"].T


# --------------------------------------------------------------- feed-forward
def dense_ff(h: np.ndarray, w: Dict[str, np.ndarray]) -> np.ndarray:
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


# ------------------------------------------------------------------ the model
def sub(tensors: Dict[str, np.ndarray], prefix: str) -> Dict[str, np.ndarray]:
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def layer_forward(x, cfg, tensors, li, carry):
    L = cfg["layers"][li]
    eps = float(cfg["norm"]["eps"])
    pre = f"l{li}."
    w, m = sub(tensors, pre + "mix."), L["mixer"]
    if L["type"] == "latent_attention":
        y = latent_attention(x, w, m, eps)
    elif L["type"] == "attention":
        y = attention(x, w, m, eps, carry)
    elif L["type"] == "delta":
        y = delta_mixer(x, w, m, eps)
    else:
        raise ValueError(L["type"])
    x = x + norm_around_zero(y, tensors[pre + "norm1"], eps)
    if L.get("mlp") is not None:
        x = x + norm_around_zero(dense_ff(x, sub(tensors, pre + "mlp.")), tensors[pre + "norm2"], eps)
    return x


def forward(cfg, tensors, tokens, want=None, layers_out: Optional[list] = None) -> np.ndarray:
    """Logits [len(want) or T, vocab] of one whole sequence."""
    eps = float(cfg["norm"]["eps"])
    x = norm_around_zero(tensors["embed"][np.asarray(tokens)], tensors["embed.norm"], eps)
    carry: dict = {}
    for li in range(len(cfg["layers"])):
        x = layer_forward(x, cfg, tensors, li, carry)
        if layers_out is not None:
            layers_out.append(x.copy())
    x = norm_around_zero(x, tensors["final.norm"], eps)
    if want is not None:
        x = x[np.asarray(want, dtype=np.int64)]
    return x @ tensors["head"].T
