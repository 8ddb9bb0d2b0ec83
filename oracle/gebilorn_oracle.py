"""Plain restatement of the Gebilorn design in numpy: one function per mechanism, no cache, no batching.

Test infrastructure only; it shares no code with the engine.  Everything is evaluated in the dtype of the
weights (the tests use float64), one whole sequence at a time: every row is recomputed from the token ids,
so nothing here can be wrong because of a page, a slot or the way a prompt was cut.

Notation: x [T, W] is the residual stream, one row per token, W the width.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional

import numpy as np


def rms(x, eps):
    """x / sqrt(mean of squares + eps) over the last axis."""
    return x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps)


def offset_norm(x, w, eps):
    """RMS norm whose weight is kept as its distance from one."""
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z**3)))


def bigram_rows(ids, buckets, mul_prev, mul_cur):
    """Row of the bigram table for every token: a hash of the pair (previous, current), the extra last row for the first token."""
    return [buckets if t == 0 else (int(ids[t - 1]) * mul_prev + int(ids[t]) * mul_cur) % buckets for t in range(len(ids))]


def rotation_frequencies(dims, base, scaling=None):
    """Radians per position of every pair; `scaling` slows long wavelengths down by `factor`, with a ramp between two bounds."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling is not None:
            factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave > original / low:
                f = f / factor
            elif wave >= original / high:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return np.array(out, np.float64)


def rotate(x, freqs):
    """x [T, heads, dim]: dimension i turns with dimension i + len(freqs); the rest passes."""
    T, n = x.shape[0], len(freqs)
    a = np.arange(T, dtype=np.float64)[:, None] * freqs[None, :]
    c, s = np.cos(a)[:, None, :].astype(x.dtype), np.sin(a)[:, None, :].astype(x.dtype)
    u, v = x[..., :n], x[..., n : 2 * n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * n :]], axis=-1)


def window_mask(T, size=None, keep_first=0):
    """[T, T] bool: token i sees itself, the size - 1 tokens in front of it and the first keep_first tokens."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    near = (i - j < size) if size is not None else np.ones((T, T), bool)
    return (j <= i) & (near | (j < keep_first))


def softmax_with_sink(s, sink=None):
    """Softmax over the last axis; `sink` joins the denominator as one more score without a value."""
    m = s.max(axis=-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.exp(s - m)
    d = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        d = d + np.exp(sink - m)
    return e / d


def masked_attention(q, k, v, scale, mask, sinks=None):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]; head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.empty((T, H, v.shape[2]), q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = np.where(mask, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        out[:, h] = softmax_with_sink(s, None if sinks is None else sinks[h]) @ v[:, g]
    return out


def short_convolution(u, w):
    """Causal, per channel: u [T, C], w [C, taps]; the last tap meets the token itself, zeros in front of the sequence."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1]), u.dtype), u], axis=0)
    return sum(padded[j : j + len(u)] * w[:, j] for j in range(taps))


def decay(z, tau):
    """sigmoid(z)^(1 / tau)."""
    return np.exp(-np.logaddexp(0.0, -z) / tau)


def gated_linear_attention(q, k, v, alpha):
    """q, k, alpha [T, H, dim], v [T, H, vdim] -> [T, H, vdim]; alpha shrinks the rows of the state before a token joins it."""
    T, H, d = k.shape
    S = np.zeros((H, d, v.shape[2]), q.dtype)
    out = np.empty((T, H, v.shape[2]), q.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def route(z, top, scale):
    """Router logits [T, E] -> (chosen [T, top], weights): softmax over all, the largest, not renormalised."""
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s = s / s.sum(axis=1, keepdims=True)
    chosen = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=1) * scale


def gated_mlp(h, gate, up, down, act):
    return (act(h @ gate.T) * (h @ up.T)) @ down.T


class Oracle:
    """config: the dict of config.json; weights: name -> array (any float dtype, widened to `dtype`)."""

    def __init__(self, config: dict, weights: Dict[str, np.ndarray], dtype=np.float64, cache_round=None):
        """cache_round: applied to what a token leaves in a paged cache, as a cache of fewer bits would (None: kept as it is)."""
        self.cache_round = cache_round or (lambda c: c)
        self.cfg = config
        self.w = {k: np.asarray(v, dtype=dtype) for k, v in weights.items()}
        self.eps = float(config["norm"]["eps"])
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

    def full_attention(self, m, p, h):
        w, T, H, G = self.w, len(h), m["heads"], m["kv_heads"]
        f = rotation_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        q = rms(rotate((h @ w[p + "q"].T).reshape(T, H, -1), f), self.eps)
        k = rms(rotate((h @ w[p + "k"].T).reshape(T, G, -1), f), self.eps)
        v = (h @ w[p + "v"].T).reshape(T, G, -1)
        mask = window_mask(T, m["mask"]["size"], m["mask"].get("keep_first") or 0)
        o = masked_attention(q, self.cache_round(k), self.cache_round(v), m["scale"], mask, w[p + "sink"])
        return (o.reshape(T, -1) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T

    def window_attention(self, m, p, h):
        w, T, H, G = self.w, len(h), m["heads"], m["kv_heads"]
        q, k, v = (short_convolution(h @ w[p + n].T + w[p + n + ".b"], w[p + n + ".conv"]) for n in "qkv")
        k, v = self.cache_round(k), self.cache_round(v)
        o = masked_attention(q.reshape(T, H, -1), k.reshape(T, G, -1), v.reshape(T, G, -1), m["scale"], window_mask(T, m["mask"]["size"]), w[p + "sink"])
        return (o * sigmoid(h @ w[p + "g"].T)[:, :, None]).reshape(T, -1) @ w[p + "o"].T

    def linear_attention(self, m, p, h):
        w, T, H = self.w, len(h), m["heads"]
        q = (h @ w[p + "q"].T).reshape(T, H, -1) * m["dim"] ** -0.5
        k, v = (h @ w[p + "k"].T).reshape(T, H, -1), (h @ w[p + "v"].T).reshape(T, H, -1)
        alpha = decay((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"], m["tau"]).reshape(T, H, -1)
        o = rms(gated_linear_attention(q, k, v, alpha), self.eps) * w[p + "norm"]
        return (o.reshape(T, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T

    def latent_attention(self, m, p, h):
        w, T, H, d, r = self.w, len(h), m["heads"], m["dim"], m["kv_rank"]
        f = rotation_frequencies(m["rot_dim"], m["rot"]["base"], m["rot"].get("scaling"))
        q = ((rms(h @ w[p + "dq"].T, self.eps) * w[p + "dq.norm"]) @ w[p + "uq"].T).reshape(T, H, -1)
        kv = h @ w[p + "dkv"].T
        c = self.cache_round(rms(kv[:, :r], self.eps) * w[p + "dkv.norm"])
        k_rot = self.cache_round(rotate(kv[:, None, r:], f))
        q = np.concatenate([q[..., :d], rotate(q[..., d:], f)], axis=-1)
        k = np.concatenate([(c @ w[p + "uk"].T).reshape(T, H, d), np.repeat(k_rot, H, axis=1)], axis=-1)
        v = (c @ w[p + "uv"].T).reshape(T, H, -1)
        return masked_attention(q, k, v, m["scale"], window_mask(T)).reshape(T, -1) @ w[p + "o"].T

    def mixer(self, i: int, h):
        spec, p = self.cfg["layers"][i], f"l{i}.mix."
        m = spec["mixer"]
        if spec["type"] == "attention":
            return self.full_attention(m, p, h)
        if spec["type"] == "latent_attention":
            return self.latent_attention(m, p, h)
        return m["left_scale"] * self.window_attention(m["left"], p + "left.", h) + m["right_scale"] * self.linear_attention(m["right"], p + "right.", h)

    def feed_forward(self, i: int, h):
        f, p, w = self.cfg["layers"][i]["mlp"], f"l{i}.mlp.", self.w
        if f["kind"] == "dense":
            return gated_mlp(h, w[p + "gate"], w[p + "up"], w[p + "down"], gelu_tanh)
        r = f["router"]
        chosen, weights = route(h @ w[p + "router"].T, r["top"], r["scale"])
        out = gated_mlp(h, w[p + "shared.gate"], w[p + "shared.up"], w[p + "shared.down"], silu) * sigmoid(h @ w[p + "shared.sg"].T)
        for e in range(r["experts"]):
            t, slot = np.nonzero(chosen == e)
            if len(t):
                out[t] += weights[t, slot][:, None] * gated_mlp(h[t], w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"], silu)
        return out

    def forward(self, ids, keep_layers: bool = False) -> np.ndarray:
        """Logits [T, vocab] of a whole sequence; with keep_layers the residual stream after every layer stays in self.layers."""
        w, b = self.w, self.cfg["embedding"]["bigram"]
        x = w["embed"][np.asarray(ids)] * self.cfg["embedding"]["scale"] + w["bigram"][bigram_rows(ids, b["buckets"], b["mul_prev"], b["mul_cur"])]
        self.layers = []
        for i, spec in enumerate(self.cfg["layers"]):
            h = offset_norm(x, w[f"l{i}.norm1"], self.eps)
            y = self.mixer(i, h)
            if spec.get("mlp") is not None:
                y = y + self.feed_forward(i, h)
            x = x + y
            if keep_layers:
                self.layers.append(x.copy())
        cap = float(self.cfg["logit_softcap"])
        return cap * np.tanh((offset_norm(x, w["final.norm"], self.eps) @ w["embed"].T) / cap)

    def greedy(self, prompt, n_new: int) -> List[int]:
        ids = list(int(t) for t in prompt)
        out = []
        for _ in range(n_new):
            row = self.forward(ids)[-1]
            best = int(len(row) - 1 - np.argmax(row[::-1]))  # ties to the highest index
            out.append(best)
            ids.append(best)
        return out
