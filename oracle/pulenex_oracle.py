"""Plain restatement of the Pulenex design in numpy: one function per mechanism, no cache, no batching.

Test infrastructure only; it shares no code with the engine.  Everything is evaluated in the dtype of the
weights (the tests use float64), one whole sequence at a time: every row is recomputed from the token ids,
so nothing here can be wrong because of a page, a slot or the way a prompt was cut.

Notation: x [T, W] is the residual stream, one row per token, W the width.
"""
from __future__ import annotations

import json
import os
from typing import Dict, List

import numpy as np


def layer_norm(x, w, eps):
    """Zero mean, unit variance (mean of the squared deviations) over the last axis, times a weight."""
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(np.square(d), axis=-1, keepdims=True) + eps) * w


def rms(x, eps):
    """x / sqrt(mean of squares + eps) over the last axis."""
    return x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps)


def unit(x, eps=1e-6):
    """x / sqrt(sum of squares + eps) over the last axis."""
    return x / np.sqrt(np.sum(np.square(x), axis=-1, keepdims=True) + eps)


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rotation_frequencies(dims, base):
    """Radians per position of every pair."""
    return float(base) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)


def _turns(T, freqs, dtype):
    a = np.arange(T, dtype=np.float64)[:, None] * freqs[None, :]
    return np.cos(a)[:, None, :].astype(dtype), np.sin(a)[:, None, :].astype(dtype)


def rotate_halves(x, freqs):
    """x [T, heads, dim]: dimension i turns with dimension i + len(freqs); the rest passes."""
    n = len(freqs)
    c, s = _turns(len(x), freqs, x.dtype)
    u, v = x[..., :n], x[..., n : 2 * n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * n :]], axis=-1)


def rotate_neighbours(x, freqs):
    """x [T, heads, dim]: dimension 2 i turns with dimension 2 i + 1; the rest passes."""
    n = len(freqs)
    c, s = _turns(len(x), freqs, x.dtype)
    y = x.copy()
    u, v = x[..., 0 : 2 * n : 2], x[..., 1 : 2 * n : 2]
    y[..., 0 : 2 * n : 2], y[..., 1 : 2 * n : 2] = u * c - v * s, v * c + u * s
    return y


def window_mask(T, size=None):
    """[T, T] bool: token i sees itself and the size - 1 tokens in front of it."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < size) if size else True)


def chunk_mask(T, size=None):
    """[T, T] bool: token i sees itself and the tokens in front of it in its own chunk of `size`."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i // size == j // size) if size else True)


def softmax(s, sink=None):
    """Softmax over the last axis; `sink` joins the denominator as one more score without a value."""
    m = s.max(axis=-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.exp(s - m)
    d = e.sum(axis=-1, keepdims=True)
    return e / (d if sink is None else d + np.exp(sink - m))


def talking_scores(q, k, scale, temp, talk):
    """q [T, H, d], k [T, G, d] -> scores [H, T, T]: head h reads key head h // (H / G), times its temperature; then every head's
    scores are a mix (a row of `talk`) of all heads'."""
    H, G = q.shape[1], k.shape[1]
    s = np.stack([(q[:, h] @ k[:, h // (H // G)].T) * (scale * temp[h]) for h in range(H)])
    return np.einsum("hg,gij->hij", talk, s)


def masked_attention(scores, v, mask, sinks=None):
    """scores [H, T, T], v [T, G, vdim] -> [T, H, vdim]."""
    H, T, _ = scores.shape
    G = v.shape[1]
    out = np.empty((T, H, v.shape[2]), v.dtype)
    for h in range(H):
        out[:, h] = softmax(np.where(mask, scores[h], -np.inf), None if sinks is None else sinks[h]) @ v[:, h // (H // G)]
    return out


def short_convolution(u, w):
    """Causal, per channel: u [T, C], w [C, taps]; the last tap meets the token itself, zeros in front of the sequence."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1]), u.dtype), u], axis=0)
    return sum(padded[j : j + len(u)] * w[:, j] for j in range(taps))


def retention(q, k, v, decay):
    """q, k [T, H, dim], v [T, H, vdim], decay [H] -> [T, H, vdim]."""
    T, H, d = k.shape
    S = np.zeros((H, d, v.shape[2]), q.dtype)
    out = np.empty((T, H, v.shape[2]), q.dtype)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def channel_decay(z, a_log):
    """z [T, H, dim], a_log [H] -> factors in (0, 1)."""
    return np.exp(-np.exp(a_log)[None, :, None] * softplus(z))


def gated_delta_rule(q, k, v, g, beta):
    """q, k, g [T, H, dim], v [T, H, vdim], beta [T, H] -> [T, H, vdim]: the state shrinks row by row, then the part of v that it does
    not give back for k joins it; the token reads what it has written."""
    T, H, d = k.shape
    S = np.zeros((H, d, v.shape[2]), q.dtype)
    out = np.empty((T, H, v.shape[2]), q.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def clamped_glu(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


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
        self.latents: Dict[int, tuple] = {}

    @classmethod
    def from_dir(cls, path: str, dtype=np.float64, **kw) -> "Oracle":
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
        return cls(cfg, weights, dtype, **kw)

    def retention_mixer(self, m, p, h):
        w, T, H = self.w, len(h), m["heads"]
        f = rotation_frequencies(m["rot"]["dims"], m["rot"]["base"])
        q = rotate_halves((h @ w[p + "q"].T).reshape(T, H, -1), f)
        k = rotate_halves((h @ w[p + "k"].T).reshape(T, H, -1), f) * m["dim"] ** -0.5
        v = (h @ w[p + "v"].T).reshape(T, H, -1)
        o = rms(retention(q, k, v, np.array(m["decay"], self.dtype)), self.eps)
        return (o.reshape(T, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T

    def chunked_attention(self, m, p, h):
        w, T, H, G = self.w, len(h), m["heads"], m["kv_heads"]
        f = rotation_frequencies(m["rot"]["dims"], m["rot"]["base"])
        q, k = (short_convolution(h @ w[p + n].T, w[p + n + ".conv"]) for n in "qk")
        q, k = q.reshape(T, H, -1), k.reshape(T, G, -1)
        s = talking_scores(rotate_neighbours(q, f), self.cache_round(rotate_neighbours(k, f)), m["scale"], w[p + "temp"], w[p + "talk"])
        o = masked_attention(s, self.cache_round(k), chunk_mask(T, m["mask"]["size"]), w[p + "sink"])
        return (o.reshape(T, -1) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T

    def delta_mixer(self, m, p, h):
        w, T, H, G = self.w, len(h), m["heads"], m["kv_heads"]
        q, k, v = (silu(short_convolution(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
        q, k = (np.repeat(unit(t.reshape(T, G, -1)), H // G, axis=1) for t in (q, k))
        g = channel_decay(((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(T, H, -1), w[p + "A_log"])
        o = gated_delta_rule(q * m["dim"] ** -0.5, k, v.reshape(T, H, -1), g, sigmoid(h @ w[p + "b"].T))
        o = (rms(o, self.eps) * w[p + "norm"]).reshape(T, -1) * sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
        return o @ w[p + "o"].T

    def latent_attention(self, i, m, p, h):
        w, T, H, d, r = self.w, len(h), m["heads"], m["dim"], m["kv_rank"]
        f = rotation_frequencies(m["rot_dim"], m["rot"]["base"])
        if m.get("kv_from") is None:
            kv = h @ w[p + "dkv"].T
            self.latents[i] = (self.cache_round(rms(kv[:, :r], self.eps) * w[p + "dkv.norm"]), self.cache_round(rotate_neighbours(kv[:, None, r:], f)))
        c, k_rot = self.latents[i if m.get("kv_from") is None else m["kv_from"]]
        q = (h @ w[p + "q"].T).reshape(T, H, -1)
        q = np.concatenate([q[..., :d], rotate_neighbours(q[..., d:], f)], axis=-1)
        k = np.concatenate([(c @ w[p + "uk"].T).reshape(T, H, d), np.repeat(k_rot, H, axis=1)], axis=-1)
        s = np.einsum("ihd,jhd->hij", q, k) * m["scale"]
        o = masked_attention(s, (c @ w[p + "uv"].T).reshape(T, H, -1), window_mask(T, m["mask"]["size"]))
        return (o * sigmoid(h @ w[p + "g"].T)[:, :, None]).reshape(T, -1) @ w[p + "o"].T

    def mixer(self, i: int, h):
        spec, p = self.cfg["layers"][i], f"l{i}.mix."
        m = spec["mixer"]
        if spec["type"] == "retention":
            return self.retention_mixer(m, p, h)
        if spec["type"] == "latent_attention":
            return self.latent_attention(i, m, p, h)
        left, right = self.chunked_attention(m["left"], p + "left.", h), self.delta_mixer(m["right"], p + "right.", h)
        return 0.5 * (rms(left, self.eps) * self.w[p + "left.out"] + rms(right, self.eps) * self.w[p + "right.out"])

    def feed_forward(self, i: int, h):
        f, p, w = self.cfg["layers"][i]["mlp"], f"l{i}.mlp.", self.w
        y = clamped_glu(h @ w[p + "gate"].T + w[p + "gate.b"], h @ w[p + "up"].T + w[p + "up.b"], f["limit"])
        return y @ w[p + "down"].T + w[p + "down.b"]

    def forward(self, ids, keep_layers: bool = False) -> np.ndarray:
        """Logits [T, vocab] of a whole sequence; with keep_layers the residual stream after every layer stays in self.layers."""
        w = self.w
        x = w["embed"][np.asarray(ids)]
        self.layers, self.latents = [], {}
        for i, spec in enumerate(self.cfg["layers"]):
            n = lambda k, t: layer_norm(t, w[f"l{i}.{k}"], self.eps)
            x = x + n("norm1b", self.mixer(i, n("norm1", x)))
            if spec.get("mlp") is not None:
                x = x + n("norm2b", self.feed_forward(i, n("norm2", x)))
            if keep_layers:
                self.layers.append(x.copy())
        return (layer_norm(x, w["final.norm"], self.eps) @ w["head"].T) * self.cfg["logit_scale"]

    def greedy(self, prompt, n_new: int) -> List[int]:
        ids = list(int(t) for t in prompt)
        out = []
        for _ in range(n_new):
            row = self.forward(ids)[-1]
            best = int(len(row) - 1 - np.argmax(row[::-1]))  # ties to the highest index
            out.append(best)
            ids.append(best)
        return out
