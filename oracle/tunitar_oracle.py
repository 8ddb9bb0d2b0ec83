"""Plain restatement of the Tunitar design in numpy: one function per mechanism, no cache, no batching.

Test infrastructure only; it shares no code with the engine.  Everything is evaluated in the dtype of the
inputs (the tests use float64), one whole sequence at a time: every row is recomputed from the token ids,
so nothing here can be wrong because of a page, a slot or the way a prompt was cut.

Notation: x [T, W] is the residual stream, one row per token, W the width.
"""
from __future__ import annotations

import json
import os
from typing import Dict, List, Optional

import numpy as np


def rms(x, eps):
    """x / sqrt(mean of squares + eps) over the last axis."""
    return x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps)


def group_norm(x, w, groups, eps):
    """The vector cut into `groups` equal runs, each divided by its own root mean square, times w."""
    T, W = x.shape
    return rms(x.reshape(T, groups, W // groups), eps).reshape(T, W) * w


def token_shift(h, mix):
    """Row t moves towards row t-1 (before its own move) by `mix` per element; row -1 is zero."""
    prev = np.zeros_like(h)
    prev[1:] = h[:-1]
    return h + (prev - h) * mix


def latents(h, w_dkv, w_norm, eps):
    """What a token leaves in the cache: the normalised down-projection [T, R]."""
    return rms(h @ w_dkv.T, eps) * w_norm


def latent_attention(h, c, w_q, w_uk, w_uv, w_g, w_o, heads, dim, vdim, scale):
    """Causal softmax attention whose keys and values are both read off the latents c [T, R]; no positions."""
    T = h.shape[0]
    q = (h @ w_q.T).reshape(T, heads, dim)
    k = (c @ w_uk.T).reshape(T, heads, dim)
    v = (c @ w_uv.T).reshape(T, heads, vdim)
    future = np.arange(T)[None, :] > np.arange(T)[:, None]
    out = np.empty((T, heads, vdim), h.dtype)
    for a in range(heads):
        s = (q[:, a] @ k[:, a].T) * scale
        s[future] = -np.inf
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, a] = (p / p.sum(axis=1, keepdims=True)) @ v[:, a]
    gate = 1.0 / (1.0 + np.exp(-(h @ w_g.T)))
    return (out.reshape(T, heads * vdim) * gate) @ w_o.T


def squared_relu_mlp(h, w_up, w_down):
    return np.square(np.maximum(h @ w_up.T, 0.0)) @ w_down.T


class Oracle:
    """config: the dict of config.json; weights: name -> array (any float dtype, widened to `dtype`)."""

    def __init__(self, config: dict, weights: Dict[str, np.ndarray], dtype=np.float64, cache_round=None):
        """cache_round: applied to the latents as a cache of fewer bits would (None: kept as they are)."""
        self.cache_round = cache_round or (lambda c: c)
        self.cfg = config
        self.w = {k: np.asarray(v, dtype=dtype) for k, v in weights.items()}
        self.groups = int(config["norm"]["groups"])
        self.eps = float(config["norm"]["eps"])
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

    def mixer(self, i: int, h, cached: Dict[int, np.ndarray]):
        m, p, w = self.cfg["layers"][i]["mixer"], f"l{i}.mix.", self.w
        src: Optional[int] = m.get("kv_from")
        if src is None:
            cached[i] = self.cache_round(latents(h, w[p + "dkv"], w[p + "dkv.norm"], self.eps))
            src = i
        return latent_attention(h, cached[src], w[p + "q"], w[p + "uk"], w[p + "uv"], w[p + "g"], w[p + "o"], m["heads"], m["dim"], m["vdim"], m["scale"])

    def forward(self, ids, keep_layers: bool = False) -> np.ndarray:
        """Logits [T, vocab] of a whole sequence; with keep_layers the residual stream after every layer stays in self.layers."""
        w = self.w
        x = w["embed"][np.asarray(ids)].copy()
        cached: Dict[int, np.ndarray] = {}
        self.layers, self.latents = [], cached
        for i, spec in enumerate(self.cfg["layers"]):
            p = f"l{i}."
            h = token_shift(group_norm(x, w[p + "norm1"], self.groups, self.eps), w[p + "shift"])
            x = x + self.mixer(i, h, cached) * w[p + "ls1"]
            if spec.get("mlp") is not None:
                h = group_norm(x, w[p + "norm2"], self.groups, self.eps)
                x = x + squared_relu_mlp(h, w[p + "mlp.up"], w[p + "mlp.down"]) * w[p + "ls2"]
            if keep_layers:
                self.layers.append(x.copy())
        return group_norm(x, w["final.norm"], self.groups, self.eps) @ w["head"].T

    def greedy(self, prompt, n_new: int) -> List[int]:
        ids = list(int(t) for t in prompt)
        out = []
        for _ in range(n_new):
            row = self.forward(ids)[-1]
            best = int(len(row) - 1 - np.argmax(row[::-1]))  # ties to the highest index
            out.append(best)
            ids.append(best)
        return out
