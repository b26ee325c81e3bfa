"""Rugezen restated plainly: one function per mechanism, float64, loops over tokens.

Nothing here is shared with the engine: weights arrive as a dict of numpy arrays by tensor name, the
configuration as the parsed ``config.json``.  Slow on purpose; the tests use small sizes.  Notation: ``x`` a row of
the residual stream, ``h`` what a sublayer reads, ``p`` a position.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional

import numpy as np


def unit_rms(x: np.ndarray, eps: float) -> np.ndarray:
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z: np.ndarray) -> np.ndarray:
    e = np.exp(-np.abs(z))
    return np.where(z >= 0.0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z: np.ndarray) -> np.ndarray:
    return z * sigmoid(z)


def rotate_pairs(v: np.ndarray, p: int, base: float, dims: int) -> np.ndarray:
    """Entries (2i, 2i+1) of the first ``dims`` turn by p * base^(-2i/dims); the rest pass."""
    out = v.copy()
    for i in range(dims // 2):
        a = p * base ** (-2.0 * i / dims)
        c, s = math.cos(a), math.sin(a)
        u, w = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i] = u * c - w * s
        out[..., 2 * i + 1] = w * c + u * s
    return out


def heads_ready(rows: np.ndarray, n: int, dim: int, rot: Optional[dict], eps: float) -> np.ndarray:
    """Projected rows [T, n * dim] -> [T, n, dim]: rotated at their positions, then each head over its root mean square."""
    T = rows.shape[0]
    heads = rows.reshape(T, n, dim)
    if rot:
        heads = np.stack([rotate_pairs(heads[t], t, float(rot["base"]), int(rot["dims"])) for t in range(T)])
    return unit_rms(heads, eps)


def softmax_plus_one(s: np.ndarray) -> np.ndarray:
    """Weights e^s_j / (1 + sum e^s_j) of one row of scores."""
    m = max(float(s.max()), 0.0)
    e = np.exp(s - m)
    return e / (math.exp(-m) + e.sum())


def capped(s: np.ndarray, cap: float) -> np.ndarray:
    return cap * np.tanh(s / cap)


def attention(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, m: dict, eps: float) -> np.ndarray:
    T = h.shape[0]
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = heads_ready(h @ w[pre + ".q"].T, H, d, m.get("rot"), eps)
    k = heads_ready(h @ w[pre + ".k"].T, G, d, m.get("rot"), eps)
    v = unit_rms((h @ w[pre + ".v"].T).reshape(T, G, vd), eps)
    out = np.zeros((T, H, vd))
    for t in range(T):
        for hd in range(H):
            g = hd // (H // G)
            s = (k[:t + 1, g] @ q[t, hd]) * float(m["scale"])
            if m.get("softcap"):
                s = capped(s, float(m["softcap"]))
            out[t, hd] = softmax_plus_one(s) @ v[:t + 1, g]
    return out.reshape(T, H * vd) @ w[pre + ".o"].T


def candidate(u: np.ndarray) -> np.ndarray:
    """u + 1/2 from zero on, sigmoid(u) below: positive everywhere, continuous at zero."""
    return np.where(u >= 0.0, u + 0.5, sigmoid(u))


def min_gru(h: np.ndarray, w: Dict[str, np.ndarray], pre: str) -> np.ndarray:
    z = sigmoid(h @ w[pre + ".z"].T + w[pre + ".z.b"])
    c = candidate(h @ w[pre + ".x"].T + w[pre + ".x.b"])
    gate = silu(h @ w[pre + ".g"].T)
    S = np.zeros(z.shape[1])
    y = np.zeros_like(z)
    for t in range(h.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * c[t]
        y[t] = S * gate[t]
    return y @ w[pre + ".o"].T


def feed_forward(h: np.ndarray, w: Dict[str, np.ndarray], pre: str) -> np.ndarray:
    a = np.maximum(h @ w[pre + ".up"].T + w[pre + ".up.b"], 0.0)
    return (a * a) @ w[pre + ".down"].T + w[pre + ".down.b"]


def layer_order(cfg: dict) -> List[int]:
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    inner = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + inner * loop["times"] + list(range(loop["stop"], n))


def layer(cfg: dict, w: Dict[str, np.ndarray], i: int, x: np.ndarray) -> np.ndarray:
    """x + m (mixer(norm1 x) + ff(norm2 x)), both of the same x."""
    spec, pre, eps = cfg["layers"][i], f"l{i}", float(cfg["norm"]["eps"])
    h = unit_rms(x, eps) * w[pre + ".norm1"]
    if spec["type"] == "attention":
        y = attention(h, w, pre + ".mix", spec["mixer"], eps)
    elif spec["type"] == "mingru":
        y = min_gru(h, w, pre + ".mix")
    else:
        raise ValueError(f"unknown layer type {spec['type']}")
    if spec.get("mlp") is not None:
        y = y + feed_forward(unit_rms(x, eps) * w[pre + ".norm2"], w, pre + ".mlp")
    return x + float(cfg["residual_mult"]) * y


def forward(cfg: dict, w: Dict[str, np.ndarray], tokens: List[int], layer_outputs: Optional[list] = None) -> np.ndarray:
    """Logits [T, vocab] of one sequence from position 0; ``layer_outputs`` collects the stream after every layer run.
    The whole sequence runs at once from nothing, so a looped layer's passes each see their own keys and state."""
    x = w["embed"][np.asarray(tokens)]
    for i in layer_order(cfg):
        x = layer(cfg, w, i, x)
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return (unit_rms(x, float(cfg["norm"]["eps"])) * w["final.norm"]) @ w["head"].T


def read_safetensors(path: str) -> Dict[str, np.ndarray]:
    """A reader of its own: 8 bytes of length, a JSON header, raw little-endian data; everything widened to float64."""
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        raw = data[a:b]
        if info["dtype"] == "BF16":
            arr = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif info["dtype"] == "F32":
            arr = np.frombuffer(raw, dtype="<f4").astype(np.float64)
        else:
            raise ValueError(f"{name}: dtype {info['dtype']} is not read here")
        out[name] = arr.reshape(info["shape"])
    return out


def greedy(cfg: dict, w: Dict[str, np.ndarray], prompt: List[int], n: int) -> List[int]:
    """n tokens after the prompt, each the first largest logit."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]


def load_folder(model_dir: str):
    with open(os.path.join(model_dir, "config.json"), "r", encoding="utf-8") as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))
