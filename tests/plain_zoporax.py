"""Zoporax restated plainly: one function per mechanism, float64, loops over tokens.

Nothing here is shared with the engine: weights arrive as a dict of numpy arrays by tensor
name, the configuration as the parsed ``config.json``.  Slow on purpose; the tests use small
sizes.  Notation: ``x`` a row of the residual stream, ``h`` what a sublayer reads, ``p`` a position.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional, Tuple

import numpy as np


def rms_norm(x: np.ndarray, weight: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu_erf(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def frequencies(rot: dict) -> Tuple[np.ndarray, float]:
    """The angle per position of each rotated pair, and what cos and sin are multiplied by."""
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return np.array(f), 1.0
    factor = float(sc["factor"])

    def dim_of(turns):
        return dims * math.log(float(sc["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim_of(float(sc["fast"]))), 0)
    hi = min(math.ceil(dim_of(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return np.array(out), 0.1 * math.log(factor) + 1.0


def rotate_halves(v: np.ndarray, p: int, rot: dict) -> np.ndarray:
    """Entry i turns with entry i + dims/2; entries past ``dims`` pass unchanged."""
    freq, mag = frequencies(rot)
    half = len(freq)
    out = v.copy()
    for i in range(half):
        c, s = mag * math.cos(p * freq[i]), mag * math.sin(p * freq[i])
        u, w = v[..., i], v[..., i + half]
        out[..., i] = u * c - w * s
        out[..., i + half] = w * c + u * s
    return out


def softmax(s: np.ndarray) -> np.ndarray:
    e = np.exp(s - s.max())
    return e / e.sum()


def first_visible(t: int, mask: Optional[dict]) -> int:
    """The oldest position that position t sees."""
    return max(0, t - int(mask["size"]) + 1) if mask else 0


def latent_attention(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, m: dict, eps: float) -> np.ndarray:
    """Queries through a latent of their own, keys and values per head from the keys' latent, one rotated key part for
    all heads, a sliding window, a sigmoid gate on every entry of the heads side by side."""
    T = h.shape[0]
    H, d, rd, vd, rank, rot = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["rot"]
    cq = rms_norm(h @ w[pre + ".dq"].T, w[pre + ".dq.norm"], eps)
    q = cq @ w[pre + ".uq"].T
    down = h @ w[pre + ".dkv"].T
    c = rms_norm(down[:, :rank], w[pre + ".dkv.norm"], eps)
    r = np.stack([rotate_halves(down[t, rank:], t, rot) for t in range(T)])
    keys, values = c @ w[pre + ".uk"].T, c @ w[pre + ".uv"].T
    heads = np.zeros((T, H * vd))
    for t in range(T):
        a = first_visible(t, m.get("mask"))
        for n in range(H):
            plain = q[t, n * (d + rd): n * (d + rd) + d]
            turned = rotate_halves(q[t, n * (d + rd) + d: (n + 1) * (d + rd)], t, rot)
            s = (keys[a:t + 1, n * d:(n + 1) * d] @ plain + r[a:t + 1] @ turned) * float(m["scale"])
            heads[t, n * vd:(n + 1) * vd] = softmax(s) @ values[a:t + 1, n * vd:(n + 1) * vd]
    return (heads * sigmoid(h @ w[pre + ".g"].T)) @ w[pre + ".o"].T


def lightning(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, m: dict, eps: float, state: Optional[np.ndarray] = None) -> np.ndarray:
    """S <- decay S + k v^T, o = S^T q per head; one norm over all heads, then the gate.  ``state`` [heads, dim, vdim] is
    updated in place when given (zero: the start of a sequence)."""
    T = h.shape[0]
    H, d, vd = m["heads"], m["dim"], m["vdim"]
    q, k, v = (silu(h @ w[f"{pre}.{n}"].T) for n in ("q", "k", "v"))
    S = np.zeros((H, d, vd)) if state is None else state
    o = np.zeros((T, H * vd))
    for t in range(T):
        for n in range(H):
            S[n] = float(m["decay"][n]) * S[n] + np.outer(k[t, n * d:(n + 1) * d], v[t, n * vd:(n + 1) * vd])
            o[t, n * vd:(n + 1) * vd] = S[n].T @ q[t, n * d:(n + 1) * d]
    return (rms_norm(o, w[pre + ".norm"], eps) * sigmoid(h @ w[pre + ".g"].T)) @ w[pre + ".o"].T


def dense_feed_forward(h: np.ndarray, w: Dict[str, np.ndarray], pre: str) -> np.ndarray:
    gate = h @ w[pre + ".gate"].T + w[pre + ".gate.b"]
    up = h @ w[pre + ".up"].T + w[pre + ".up.b"]
    return (gelu_tanh(gate) * up) @ w[pre + ".down"].T + w[pre + ".down.b"]


def expert(h: np.ndarray, w: Dict[str, np.ndarray], pre: str) -> np.ndarray:
    return gelu_erf(h @ w[pre + ".up"].T) @ w[pre + ".down"].T


def kept_experts(scores: np.ndarray, groups: Optional[dict]) -> List[int]:
    """The experts of the best groups, a group's score being the sum of its two largest scores."""
    n = len(scores)
    if not groups:
        return list(range(n))
    per = n // int(groups["count"])
    rank = []
    for g in range(int(groups["count"])):
        best = sorted(scores[g * per:(g + 1) * per], reverse=True)[:2]
        rank.append((-sum(best), g))
    keep = sorted(g for _, g in sorted(rank)[:int(groups["keep"])])
    return [g * per + i for g in keep for i in range(per)]


def route(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, ff: dict):
    """Per row: the chosen experts and their weights (the scores over their sum, times the router's scale)."""
    router = ff["router"]
    s = sigmoid(h @ w[pre + ".router"].T)
    picks, weights = [], []
    for row in s:
        can = kept_experts(row, router.get("groups"))
        chosen = sorted(can, key=lambda e: (-row[e], e))[:int(router["top"])]
        total = sum(row[e] for e in chosen) + 1e-20
        picks.append(chosen)
        weights.append([row[e] / total * float(router.get("scale", 1.0)) for e in chosen])
    return picks, weights


def routed_feed_forward(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, ff: dict, picks_out: Optional[dict] = None) -> np.ndarray:
    picks, weights = route(h, w, pre, ff)
    if picks_out is not None:
        picks_out[pre] = picks
    out = np.zeros((h.shape[0], w[pre + ".e0.down"].shape[0]))
    for e in range(int(ff["router"]["experts"])):
        rows = [t for t in range(h.shape[0]) if e in picks[t]]
        if rows:
            y = expert(h[rows], w, f"{pre}.e{e}")
            for t, row in zip(rows, y):
                out[t] += weights[t][picks[t].index(e)] * row
    if ff.get("shared"):
        out += sigmoid(h @ w[pre + ".shared.sg"].T) * expert(h, w, pre + ".shared")
    return out


MIXERS = {"latent_attention": latent_attention, "lightning": lightning}


def forward(cfg: dict, w: Dict[str, np.ndarray], tokens: List[int], layer_outputs: Optional[list] = None,
            picks: Optional[dict] = None) -> np.ndarray:
    """Logits [T, vocab] of one sequence from position 0; ``layer_outputs`` collects the stream after every layer,
    ``picks`` the chosen experts of every routed feed-forward by its tensor-name prefix."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][np.asarray(tokens)].copy()
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}"
        x = x + MIXERS[layer["type"]](rms_norm(x, w[pre + ".norm1"], eps), w, pre + ".mix", layer["mixer"], eps)
        ff = layer.get("mlp")
        if ff is not None:
            h = rms_norm(x, w[pre + ".norm2"], eps)
            x = x + (dense_feed_forward(h, w, pre + ".mlp") if ff["kind"] == "dense" else routed_feed_forward(h, w, pre + ".mlp", ff, picks))
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy(cfg: dict, w: Dict[str, np.ndarray], prompt: List[int], n: int) -> List[int]:
    """n tokens after the prompt, each the first largest logit."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]


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


def load_folder(model_dir: str):
    with open(os.path.join(model_dir, "config.json"), "r", encoding="utf-8") as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))
