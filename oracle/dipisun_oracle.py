"""Plain restatement of the Dipisun design in numpy: one function per mechanism, no cache, no batching.

Test infrastructure only; it shares no code with the engine.  Everything is evaluated in the dtype of the
weights (the tests use float64), one whole sequence at a time: every row is recomputed from the token ids,
so nothing here can be wrong because of a page, a slot or the way a prompt was cut.

Notation: x [T, W] is the residual stream, one row per token, W the width.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List

import numpy as np


def rms(x, eps):
    """x / sqrt(mean of squares + eps) over the last axis."""
    return x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps)


def position_vectors(positions, width, dtype=np.float64):
    """[T, width]: sine in the even and cosine in the odd elements, pair i turning by 10000^(-2 i / width) per position."""
    p = np.asarray(positions, np.float64)[:, None]
    e = np.arange(width)
    angle = p * 10000.0 ** (-(e - e % 2) / width)[None, :]
    return np.where(e % 2 == 0, np.sin(angle), np.cos(angle)).astype(dtype)


def temperature(positions, coef, every):
    """Factor of the queries: grows with the logarithm of how many times `every` tokens have passed."""
    return np.array([1.0 + coef * math.log((int(p) + 1) // every + 1) for p in positions])


def distance_bucket(n, buckets, reach):
    """Row of the bias table for a key n tokens back: one row per distance up to half the table, logarithmic steps up to `reach`."""
    half = buckets // 2
    if n < half:
        return n
    if n >= reach:
        return buckets - 1
    # the small term keeps a distance that lies exactly on a step on its upper side
    return min(buckets - 1, half + int(math.floor(math.log(n / half) / math.log(reach / half) * (buckets - half) + 1e-9)))


def distance_bias(table, T, reach):
    """[T, T, heads] bias of query i on key j (zero where j > i); table [buckets, heads]."""
    rows = table[[distance_bucket(n, table.shape[0], reach) for n in range(T)]]
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return np.where((j <= i)[..., None], rows[np.maximum(i - j, 0)], 0.0)


def norm_all_heads(q, w, eps):
    """One root mean square over the whole projection [T, heads * dim]."""
    return rms(q, eps) * w


def norm_each_head(q, w, heads, eps):
    """Every head by its own root mean square; one weight vector for all heads."""
    T = q.shape[0]
    return (rms(q.reshape(T, heads, -1), eps) * w).reshape(T, -1)


def blend_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def grouped_attention(q, k, v, heads, kv_heads, scale, bias=None):
    """Causal softmax attention; q [T, heads * dim], k [T, kv_heads * dim], v [T, kv_heads * vdim] -> [T, heads * vdim]."""
    T = q.shape[0]
    q, k, v = q.reshape(T, heads, -1), k.reshape(T, kv_heads, -1), v.reshape(T, kv_heads, -1)
    future = np.arange(T)[None, :] > np.arange(T)[:, None]
    out = np.empty((T, heads, v.shape[2]), q.dtype)
    for h in range(heads):
        g = h // (heads // kv_heads)
        s = (q[:, h] @ k[:, g].T) * scale
        if bias is not None:
            s = s + bias[:, :, h]
        s[future] = -np.inf
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, g]
    return out.reshape(T, -1)


def route(z, correction, top):
    """Router logits z [T, E] -> (chosen [T, top], weights [T, top]): softmax scores, chosen by score + correction."""
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s = s / s.sum(axis=1, keepdims=True)
    chosen = np.argsort(-(s + correction), axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=1)


def clamped_expert(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0)) @ down.T


def mixture(h, w_router, correction, top, experts):
    """experts: one function [n, W] -> [n, W] per router output, identity experts included."""
    chosen, weights = route(h @ w_router.T, correction, top)
    out = np.zeros_like(h)
    for e in range(len(experts)):
        t, slot = np.nonzero(chosen == e)
        if len(t):
            out[t] += weights[t, slot][:, None] * experts[e](h[t])
    return out


class Oracle:
    """config: the dict of config.json; weights: name -> array (any float dtype, widened to `dtype`)."""

    def __init__(self, config: dict, weights: Dict[str, np.ndarray], dtype=np.float64, cache_round=None):
        """cache_round: applied to keys and values as a cache of fewer bits would (None: kept as they are)."""
        self.cache_round = cache_round or (lambda c: c)
        self.cfg = config
        self.w = {k: np.asarray(v, dtype=dtype) for k, v in weights.items()}
        self.eps = float(config["norm"]["eps"])
        self.mult = float(config["residual_mult"])
        self.dtype = dtype
        self.layers: List[np.ndarray] = []

    @classmethod
    def from_dir(cls, path: str, dtype=np.float64) -> "Oracle":
        with open(os.path.join(path, "config.json")) as f:
            cfg = json.load(f)
        with open(os.path.join(path, "model.safetensors"), "rb") as f:
            n = int.from_bytes(f.read(8), "little")
            head = json.loads(f.read(n))
            blob = f.read()
        weights = {}
        for name, t in head.items():
            if name == "__metadata__":
                continue
            lo, hi = t["data_offsets"]
            raw = np.frombuffer(blob[lo:hi], np.uint16 if t["dtype"] == "BF16" else np.float32)
            if t["dtype"] == "BF16":
                raw = (raw.astype(np.uint32) << 16).view(np.float32)
            weights[name] = raw.reshape(t["shape"])
        return cls(cfg, weights, dtype)

    def mixer(self, i: int, h, cached: Dict[int, tuple], first: Dict[int, np.ndarray]):
        spec, p, w = self.cfg["layers"][i], f"l{i}.mix.", self.w
        m = spec["mixer"]
        q, k, v = h @ w[p + "q"].T, h @ w[p + "k"].T, h @ w[p + "v"].T
        bias = None
        if spec["type"] == "attention":
            q, k = norm_all_heads(q, w[p + "q.norm"], self.eps), norm_all_heads(k, w[p + "k.norm"], self.eps)
            if m.get("q_temp"):
                q = q * temperature(range(len(h)), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None].astype(self.dtype)
            bias = distance_bias(w[p + "rel"], len(h), m["bias_max"])
        else:
            q, k = norm_each_head(q, w[p + "q.norm"], m["heads"], self.eps), norm_each_head(k, w[p + "k.norm"], m["kv_heads"], self.eps)
        if m.get("v_mix"):
            if "v" in first:
                v = blend_values(v, first["v"], w[p + "vmix"].reshape(()))
            else:
                first["v"] = v
        cached[i] = self.cache_round(k), self.cache_round(v)
        return grouped_attention(q, *cached[i], m["heads"], m["kv_heads"], m["scale"], bias) @ w[p + "o"].T

    def feed_forward(self, i: int, h):
        f, p, w = self.cfg["layers"][i]["mlp"], f"l{i}.mlp.", self.w
        r = f["router"]
        experts = [lambda t, e=e: clamped_expert(t, w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"], f["expert"]["limit"]) for e in range(r["experts"])]
        experts += [lambda t: t] * (r.get("identity") or 0)
        return mixture(h, w[p + "router"], w[p + "correction"], r["top"], experts)

    def forward(self, ids, keep_layers: bool = False) -> np.ndarray:
        """Logits [T, vocab] of a whole sequence; with keep_layers the residual stream after every layer stays in self.layers."""
        w = self.w
        x = w["embed"][np.asarray(ids)] + position_vectors(range(len(ids)), self.cfg["width"], self.dtype)
        cached: Dict[int, tuple] = {}
        first: Dict[int, np.ndarray] = {}
        self.layers, self.cached = [], cached
        for i, spec in enumerate(self.cfg["layers"]):
            p = f"l{i}."
            x = x + self.mult * rms(self.mixer(i, x, cached, first), self.eps) * w[p + "norm1"]
            if spec.get("mlp") is not None:
                x = x + self.mult * rms(self.feed_forward(i, x), self.eps) * w[p + "norm2"]
            if keep_layers:
                self.layers.append(x.copy())
        return rms(x, self.eps) * w["final.norm"] @ w["head"].T

    def greedy(self, prompt, n_new: int) -> List[int]:
        ids = list(int(t) for t in prompt)
        out = []
        for _ in range(n_new):
            row = self.forward(ids)[-1]
            best = int(len(row) - 1 - np.argmax(row[::-1]))  # ties to the highest index
            out.append(best)
            ids.append(best)
        return out
