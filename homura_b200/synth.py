"""Seeded synthetic checkpoints in the two container formats Homura loads.

There are no real checkpoints where this code runs, so tests and the benchmark write
random-initialised models of the named architectures from a seed:

* ``write_hf_model``  -> ``config.json`` + ``model.safetensors`` with the HuggingFace tensor
  names that Homura's loader expects (src/hf/weights.rs:267-417 in the Homura repository):
  linears stored ``[out, in]`` in bf16 ~N(0, 0.02) rounded to nearest even, norms = 1,
  biases ~N(0, 0.02).
* ``write_gguf_model`` -> a GGUF v3 file with ``blk.N.*`` tensors (src/gguf.rs:589-708):
  Q8_0 or Q4_0 blocks for all linears (f16 scale = |N(0, 0.01)|, codes uniform), bf16
  embedding and norms.

Every tensor draws from its own PCG64 stream keyed by (seed, crc32(name)), so the bytes do
not depend on generation order.
"""
from __future__ import annotations

import json
import os
import struct
import zlib
from dataclasses import dataclass, asdict
from typing import Dict, Iterable, List, Optional, Tuple

import numpy as np

GGUF_MAGIC = 0x46554747  # "GGUF" little-endian
GGML_F32, GGML_F16, GGML_Q4_0, GGML_Q8_0, GGML_BF16 = 0, 1, 2, 8, 30
GGML_Q4_K, GGML_Q6_K = 12, 14


@dataclass
class DecoderConfig:
    """Mirror of Homura's TransformerConfig (src/hf/config.rs:11-38)."""

    hidden_size: int
    intermediate_size: int
    num_attention_heads: int
    num_hidden_layers: int
    num_key_value_heads: int
    vocab_size: int
    rms_norm_eps: float = 1e-6
    rope_theta: float = 10000.0
    max_position_embeddings: int = 2048
    tie_word_embeddings: bool = False
    head_dim: Optional[int] = None
    # model-shape facts Homura infers from tensor names, not from config.json
    qkv_bias: bool = False
    qk_norm: bool = False

    @property
    def hd(self) -> int:
        return self.head_dim or self.hidden_size // self.num_attention_heads

    @property
    def q_dim(self) -> int:
        return self.num_attention_heads * self.hd

    @property
    def kv_dim(self) -> int:
        return self.num_key_value_heads * self.hd


# Architectures named by the benchmark configurations.
QWEN25_05B = DecoderConfig(896, 4864, 14, 24, 2, 151936, 1e-6, 1e6, 2048, True, None, True, False)
QWEN25_15B = DecoderConfig(1536, 8960, 12, 28, 2, 151936, 1e-6, 1e6, 2048, True, None, True, False)
QWEN3_06B = DecoderConfig(1024, 3072, 16, 28, 8, 151936, 1e-6, 1e6, 2048, True, 128, False, True)
TINYLLAMA_11B = DecoderConfig(2048, 5632, 32, 22, 4, 32000, 1e-5, 1e4, 2048, False, None, False, False)


def tiny_config(**kw) -> DecoderConfig:
    """A small Qwen2-shaped model for tests that the CPU oracle runs in milliseconds."""
    base = dict(
        hidden_size=256,
        intermediate_size=640,
        num_attention_heads=4,
        num_hidden_layers=3,
        num_key_value_heads=2,
        vocab_size=1024,
        rms_norm_eps=1e-6,
        rope_theta=1e6,
        max_position_embeddings=256,
        tie_word_embeddings=True,
        head_dim=None,
        qkv_bias=True,
        qk_norm=False,
    )
    base.update(kw)
    return DecoderConfig(**base)


def _rng(seed: int, name: str) -> np.random.Generator:
    return np.random.Generator(np.random.PCG64([seed, zlib.crc32(name.encode())]))


def f32_to_bf16_rne(x: np.ndarray) -> np.ndarray:
    """float32 -> bf16 bit patterns (uint16), round to nearest even."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    rounded = u + (np.uint32(0x7FFF) + ((u >> np.uint32(16)) & np.uint32(1)))
    return (rounded >> np.uint32(16)).astype(np.uint16)


def bf16_to_f32(b: np.ndarray) -> np.ndarray:
    return (b.astype(np.uint32) << np.uint32(16)).view(np.float32)


def normal_bf16(seed: int, name: str, shape: Tuple[int, ...], std: float = 0.02) -> np.ndarray:
    g = _rng(seed, name)
    n = int(np.prod(shape))
    out = np.empty(n, dtype=np.uint16)
    step = 1 << 24
    for i in range(0, n, step):
        m = min(step, n - i)
        v = g.standard_normal(m, dtype=np.float32)
        v *= np.float32(std)
        out[i : i + m] = f32_to_bf16_rne(v)
    return out.reshape(shape)


def ones_bf16(shape) -> np.ndarray:
    return np.full(shape, 0x3F80, dtype=np.uint16)


def hf_tensor_specs(cfg: DecoderConfig) -> List[Tuple[str, Tuple[int, ...], str]]:
    """(name, shape, kind) in file order; kind in {'w','one','bias'}."""
    H, I, V = cfg.hidden_size, cfg.intermediate_size, cfg.vocab_size
    specs: List[Tuple[str, Tuple[int, ...], str]] = [("model.embed_tokens.weight", (V, H), "w")]
    for i in range(cfg.num_hidden_layers):
        p = f"model.layers.{i}."
        specs.append((p + "input_layernorm.weight", (H,), "one"))
        for nm, out_f in (("q", cfg.q_dim), ("k", cfg.kv_dim), ("v", cfg.kv_dim)):
            specs.append((p + f"self_attn.{nm}_proj.weight", (out_f, H), "w"))
            if cfg.qkv_bias:
                specs.append((p + f"self_attn.{nm}_proj.bias", (out_f,), "bias"))
        if cfg.qk_norm:
            specs.append((p + "self_attn.q_norm.weight", (cfg.hd,), "one"))
            specs.append((p + "self_attn.k_norm.weight", (cfg.hd,), "one"))
        specs.append((p + "self_attn.o_proj.weight", (H, cfg.q_dim), "w"))
        specs.append((p + "post_attention_layernorm.weight", (H,), "one"))
        specs.append((p + "mlp.gate_proj.weight", (I, H), "w"))
        specs.append((p + "mlp.up_proj.weight", (I, H), "w"))
        specs.append((p + "mlp.down_proj.weight", (H, I), "w"))
    specs.append(("model.norm.weight", (H,), "one"))
    if not cfg.tie_word_embeddings:
        specs.append(("lm_head.weight", (V, H), "w"))
    return specs


def config_json(cfg: DecoderConfig) -> dict:
    d = {
        "hidden_size": cfg.hidden_size,
        "intermediate_size": cfg.intermediate_size,
        "num_attention_heads": cfg.num_attention_heads,
        "num_hidden_layers": cfg.num_hidden_layers,
        "num_key_value_heads": cfg.num_key_value_heads,
        "vocab_size": cfg.vocab_size,
        "rms_norm_eps": cfg.rms_norm_eps,
        "rope_theta": cfg.rope_theta,
        "max_position_embeddings": cfg.max_position_embeddings,
        "tie_word_embeddings": cfg.tie_word_embeddings,
    }
    if cfg.head_dim is not None:
        d["head_dim"] = cfg.head_dim
    # eos_token_id is left out on purpose: it then resolves to u32::MAX in Homura
    # (src/hf/model.rs:373-377) and a random-weight run never stops early.
    return d


def write_hf_model(model_dir: str, cfg: DecoderConfig, seed: int, norm_jitter: float = 0.0) -> str:
    """Write config.json + model.safetensors (all tensors bf16).  Returns model_dir.

    ``norm_jitter`` > 0 perturbs the norm weights around 1 so tests can tell a missing
    norm multiply from a present one; the benchmark models use exactly 1.
    """

    def make(spec):
        name, shape, kind = spec
        if kind in ("w", "bias"):
            return normal_bf16(seed, name, shape, 0.02)
        if norm_jitter > 0:
            v = 1.0 + norm_jitter * _rng(seed, name).standard_normal(shape, dtype=np.float32)
            return f32_to_bf16_rne(v)
        return ones_bf16(shape)

    return _write_model(model_dir, config_json(cfg), hf_tensor_specs(cfg), make)


def _write_model(model_dir: str, config: dict, specs, make) -> str:
    """config.json + model.safetensors with every tensor in bf16; make(spec) returns the bits of one."""
    os.makedirs(model_dir, exist_ok=True)
    with open(os.path.join(model_dir, "config.json"), "w") as f:
        json.dump(config, f, indent=1)
    header: Dict[str, dict] = {}
    off = 0
    for name, shape, _ in specs:
        nbytes = int(np.prod(shape)) * 2
        header[name] = {"dtype": "BF16", "shape": list(shape), "data_offsets": [off, off + nbytes]}
        off += nbytes
    hjson = json.dumps(header, separators=(",", ":")).encode()
    hjson += b" " * ((8 - len(hjson) % 8) % 8)
    path = os.path.join(model_dir, "model.safetensors")

    # every tensor has its own generator (seed, name), so they can be drawn by several threads (numpy's
    # generators release the GIL) and still be written in file order
    from concurrent.futures import ThreadPoolExecutor

    with open(path, "wb") as f, ThreadPoolExecutor(max_workers=min(16, os.cpu_count() or 1)) as pool:
        f.write(struct.pack("<Q", len(hjson)))
        f.write(hjson)
        window = 32
        futs = [pool.submit(make, sp) for sp in specs[:window]]
        for i in range(len(specs)):
            arr = futs[i].result()
            futs[i] = None
            if i + window < len(specs):
                futs.append(pool.submit(make, specs[i + window]))
            f.write(arr.tobytes())
    return model_dir


# ---- Tunitar ----------------------------------------------------------------------------------


def tunitar_layer(heads: int, dim: int, vdim: int, kv_rank: int, ff: Optional[int], kv_from: Optional[int] = None, scale: Optional[float] = None) -> dict:
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": dim**-0.5 if scale is None else scale}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def tunitar_config(width: int, vocab: int, layers: List[dict], groups: int = 1, eps: float = 1e-6, **extra) -> dict:
    return {"architecture": "Tunitar", "width": width, "vocab": vocab, "norm": {"groups": groups, "eps": eps}, "layers": layers, **extra}


def tunitar_uniform(width: int, vocab: int, n_layers: int, heads: int, dim: int, kv_rank: int, ff: int, groups: int, share: bool = True) -> dict:
    """A stack of equal layers; with `share` every second layer reads the latents of the one in front of it."""
    return tunitar_config(width, vocab, [tunitar_layer(heads, dim, dim, kv_rank, ff, i - 1 if share and i % 2 else None) for i in range(n_layers)], groups)


# Tunitar stacks with the width, depth, heads, cache bytes per token and MLP parameters of the Qwen2.5 architectures above.
TUNITAR_05B = tunitar_uniform(896, 151936, 24, 14, 64, 256, 7296, 7)
TUNITAR_15B = tunitar_uniform(1536, 151936, 28, 12, 128, 512, 13440, 12)


def tunitar_tensor_specs(cfg: dict) -> List[Tuple[str, Tuple[int, ...], str]]:
    """(name, shape, kind); kind in {'embed', 'w', 'one', 'blend'}."""
    W, V = cfg["width"], cfg["vocab"]
    specs: List[Tuple[str, Tuple[int, ...], str]] = [("embed", (V, W), "embed")]
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q, v, r = m["heads"] * m["dim"], m["heads"] * m["vdim"], m["kv_rank"]
        specs += [(p + "norm1", (W,), "one"), (p + "mix.q", (q, W), "w")]
        if m.get("kv_from") is None:
            specs += [(p + "mix.dkv", (r, W), "w"), (p + "mix.dkv.norm", (r,), "one")]
        specs += [(p + "mix.uk", (q, r), "w"), (p + "mix.uv", (v, r), "w"), (p + "mix.g", (v, W), "w"), (p + "mix.o", (W, v), "w"), (p + "ls1", (W,), "one"), (p + "shift", (W,), "blend")]
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            specs += [(p + "norm2", (W,), "one"), (p + "mlp.up", (ff, W), "w"), (p + "mlp.down", (W, ff), "w"), (p + "ls2", (W,), "one")]
    return specs + [("final.norm", (W,), "one"), ("head", (V, W), "w")]


def tunitar_tensor(seed: int, spec) -> np.ndarray:
    """bf16 bits of one tensor: linears N(0, 1/in), vectors around 1, blends uniform in [0, 1)."""
    name, shape, kind = spec
    if kind == "w":
        return normal_bf16(seed, name, shape, float(shape[1]) ** -0.5)
    if kind == "embed":
        return normal_bf16(seed, name, shape, 1.0)
    g = _rng(seed, name)
    v = g.random(shape, dtype=np.float32) if kind == "blend" else 1.0 + 0.25 * g.standard_normal(shape, dtype=np.float32)
    return f32_to_bf16_rne(v)


def tunitar_weights(cfg: dict, seed: int) -> Dict[str, np.ndarray]:
    """name -> bf16 bits of every tensor."""
    return {s[0]: tunitar_tensor(seed, s) for s in tunitar_tensor_specs(cfg)}


def write_tunitar_model(model_dir: str, cfg: dict, seed: int, weights: Optional[Dict[str, np.ndarray]] = None) -> str:
    """config.json + model.safetensors of a Tunitar model (weights: bits to write instead of the seeded ones)."""
    return _write_model(model_dir, cfg, tunitar_tensor_specs(cfg), lambda s: tunitar_tensor(seed, s) if weights is None else weights[s[0]])


# ---- Dipisun ----------------------------------------------------------------------------------


def dipisun_mixer(heads: int, kv_heads: int, dim: int, vdim: int, reach: Optional[float] = None, temp: Optional[Tuple[float, int]] = None, v_mix: bool = False, scale: Optional[float] = None) -> dict:
    """(type, mixer).  With `reach` the kind of attention that knows distances (and may have a query temperature), else the other."""
    m: dict = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim**-0.5 if scale is None else scale, "v_mix": v_mix}
    if reach is not None:
        m["bias_max"] = reach
        if temp is not None:
            m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention_2" if reach is None else "attention", "mixer": m}


def dipisun_layer(mixer: dict, ff: Optional[int] = None, experts: int = 1, identity: int = 0, top: int = 1, limit: float = 2.0) -> dict:
    """One entry of the layer list; ff None: without a mixture."""
    mlp = None if ff is None else {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "identity": identity, "top": top}}
    return {**mixer, "mlp": mlp}


def dipisun_config(width: int, vocab: int, layers: List[dict], mult: float = 0.4, eps: float = 1e-6, **extra) -> dict:
    return {"architecture": "Dipisun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers, **extra}


def dipisun_uniform(width: int, vocab: int, n_layers: int, heads: int, kv_heads: int, dim: int, ff: int, experts: int, top: int, identity: int) -> dict:
    """Every third layer knows distances, all blend their values, all have a mixture."""
    mix = [dipisun_mixer(heads, kv_heads, dim, dim, 1024 if i % 3 == 1 else None, (0.1, 512) if i % 3 == 1 else None, True) for i in range(n_layers)]
    return dipisun_config(width, vocab, [dipisun_layer(m, ff, experts, identity, top) for m in mix], 0.25)


# Dipisun stacks with the width, depth, heads and head size of the Qwen2.5 architectures above; the chosen experts of a token have the
# MLP parameters of theirs (4 x 1216 = 4864, 8 x 1120 = 8960).
DIPISUN_05B = dipisun_uniform(896, 151936, 24, 14, 2, 64, 1216, 16, 4, 0)
DIPISUN_15B = dipisun_uniform(1536, 151936, 28, 12, 2, 128, 1120, 32, 8, 2)


def dipisun_tensor_specs(cfg: dict, buckets: int = 32) -> List[Tuple[str, Tuple[int, ...], str]]:
    """(name, shape, kind); buckets: rows of the distance tables."""
    W, V = cfg["width"], cfg["vocab"]
    specs: List[Tuple[str, Tuple[int, ...], str]] = [("embed", (V, W), "embed")]
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q, k, v, o = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]
        whole = layer["type"] == "attention"
        specs += [(p + "mix.q", (q, W), "w"), (p + "mix.k", (k, W), "w"), (p + "mix.v", (v, W), "w"), (p + "mix.o", (W, o), "w")]
        specs += [(p + "mix.q.norm", (q if whole else m["dim"],), "one"), (p + "mix.k.norm", (k if whole else m["dim"],), "one"), (p + "norm1", (W,), "one")]
        if whole:
            specs.append((p + "mix.rel", (buckets, m["heads"]), "embed"))
        if m.get("v_mix"):
            specs.append((p + "mix.vmix", (), "share"))
        if layer.get("mlp") is not None:
            f, r = layer["mlp"]["expert"]["ff"], layer["mlp"]["router"]
            n = r["experts"] + r["identity"]
            specs += [(p + "norm2", (W,), "one"), (p + "mlp.router", (n, W), "w"), (p + "mlp.correction", (n,), "small")]
            for e in range(r["experts"]):
                specs += [(f"{p}mlp.e{e}.gate", (f, W), "w"), (f"{p}mlp.e{e}.up", (f, W), "w"), (f"{p}mlp.e{e}.down", (W, f), "w")]
    return specs + [("final.norm", (W,), "one"), ("head", (V, W), "w")]


def dipisun_tensor(seed: int, spec) -> np.ndarray:
    """bf16 bits of one tensor: linears N(0, 1/in), vectors around 1, shares around one half, corrections around 0."""
    name, shape, kind = spec
    if kind in ("small", "share"):
        g = _rng(seed, name)
        v = 0.05 * g.standard_normal(shape, dtype=np.float32) if kind == "small" else 0.25 + 0.5 * g.random(shape, dtype=np.float32)
        return f32_to_bf16_rne(np.asarray(v, np.float32))
    return tunitar_tensor(seed, spec)


def dipisun_weights(cfg: dict, seed: int, buckets: int = 32) -> Dict[str, np.ndarray]:
    """name -> bf16 bits of every tensor."""
    return {s[0]: dipisun_tensor(seed, s) for s in dipisun_tensor_specs(cfg, buckets)}


def write_dipisun_model(model_dir: str, cfg: dict, seed: int, weights: Optional[Dict[str, np.ndarray]] = None, buckets: int = 32) -> str:
    """config.json + model.safetensors of a Dipisun model (weights: bits to write instead of the seeded ones)."""
    return _write_model(model_dir, cfg, dipisun_tensor_specs(cfg, buckets), lambda s: dipisun_tensor(seed, s) if weights is None else weights[s[0]])


# ---- Gebilorn ---------------------------------------------------------------------------------


def gebilorn_rot(dims: int, base: float = 10000.0, scaling: Optional[Tuple[float, float, float, float]] = None) -> dict:
    """scaling: (factor, low, high, original)."""
    r: dict = {"dims": dims, "base": base}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def gebilorn_attention(heads: int, kv_heads: int, dim: int, vdim: int, window: int, rot: dict, keep_first: int = 0, scale: Optional[float] = None) -> dict:
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim**-0.5 if scale is None else scale, "mask": {"size": window, "keep_first": keep_first}, "rot": rot}
    return {"type": "attention", "mixer": m}


def gebilorn_parallel(left: Tuple[int, int, int, int], window: int, conv: int, right: Tuple[int, int, int], tau: float = 16.0, scales: Tuple[float, float] = (1.0, 1.0), scale: Optional[float] = None) -> dict:
    """left: heads, kv_heads, dim, vdim of the windowed attention; right: heads, dim, vdim of the linear one."""
    h, g, d, v = left
    a = {"heads": h, "kv_heads": g, "dim": d, "vdim": v, "scale": d**-0.5 if scale is None else scale, "mask": {"size": window}, "conv": conv}
    return {"type": "parallel", "mixer": {"left": a, "right": dict(zip(("heads", "dim", "vdim"), right), tau=tau), "left_scale": scales[0], "right_scale": scales[1]}}


def gebilorn_latent(heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int, rot: Optional[dict] = None, scale: Optional[float] = None) -> dict:
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale, "rot": rot or gebilorn_rot(rot_dim)}
    return {"type": "latent_attention", "mixer": m}


def gebilorn_dense(ff: int) -> dict:
    return {"kind": "dense", "ff": ff}


def gebilorn_moe(ff: int, experts: int, top: int, shared_ff: int, scale: float = 1.0) -> dict:
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}, "shared": {"ff": shared_ff}}


def gebilorn_config(width: int, vocab: int, layers: List[Tuple[dict, Optional[dict]]], buckets: int = 61, muls: Tuple[int, int] = (31, 7), scale: float = 2.0, softcap: float = 50.0, eps: float = 1e-6, **extra) -> dict:
    """layers: (mixer, mlp or None) pairs."""
    emb = {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": muls[0], "mul_cur": muls[1]}}
    return {"architecture": "Gebilorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": emb, "logit_softcap": softcap, "layers": [{**m, "mlp": f} for m, f in layers], **extra}


def gebilorn_uniform(width: int, vocab: int, n_layers: int, heads: int, kv_heads: int, dim: int, ff: int, experts: int, top: int, expert_ff: int, kv_rank: int) -> dict:
    """Of every six layers four run windowed attention beside linear attention, one latent attention, one windowed attention with rotation;
    every third feed-forward is dense, the others are mixtures whose chosen and shared experts have as many parameters."""
    layers = []
    for i in range(n_layers):
        if i % 6 == 3:
            m = gebilorn_attention(heads, kv_heads, dim, dim, 1024, gebilorn_rot(dim // 2, 500000.0, (8.0, 1.0, 4.0, 8192.0)), 64)
        elif i % 6 == 5:
            m = gebilorn_latent(heads, dim, 64, dim, width // 2, kv_rank)
        else:
            m = gebilorn_parallel((heads, kv_heads, dim, dim), 512, 4, (heads, dim, dim))
        layers.append((m, gebilorn_dense(ff) if i % 3 == 0 else gebilorn_moe(expert_ff, experts, top, ff - top * expert_ff)))
    return gebilorn_config(width, vocab, layers, 65521, (8191, 131))


# Gebilorn stacks with the width, depth, heads and head size of the Qwen2.5 architectures above; dense feed-forwards, and chosen and shared
# experts together, have the MLP parameters of theirs.
GEBILORN_05B = gebilorn_uniform(896, 151936, 24, 14, 2, 64, 4864, 16, 4, 960, 256)
GEBILORN_15B = gebilorn_uniform(1536, 151936, 28, 12, 2, 128, 8960, 32, 8, 960, 512)


def gebilorn_tensor_specs(cfg: dict, decay_rank: int = 16) -> List[Tuple[str, Tuple[int, ...], str]]:
    """(name, shape, kind); decay_rank: width of the decays' latents."""
    W, V = cfg["width"], cfg["vocab"]
    specs: List[Tuple[str, Tuple[int, ...], str]] = [("embed", (V, W), "embed"), ("bigram", (cfg["embedding"]["bigram"]["buckets"] + 1, W), "embed")]

    def attention(p, m, gate):
        q, k, v, o = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]
        return [(p + "q", (q, W), "w"), (p + "k", (k, W), "w"), (p + "v", (v, W), "w"), (p + "sink", (m["heads"],), "embed"), (p + "g", (gate, W), "w"), (p + "o", (W, o), "w")]

    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        specs.append((p + "norm1", (W,), "zero"))
        if layer["type"] == "attention":
            specs += attention(p + "mix.", m, m["heads"] * m["vdim"])
        elif layer["type"] == "parallel":
            a, r = m["left"], m["right"]
            specs += attention(p + "mix.left.", a, a["heads"])
            for t, n in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                specs.append((f"{p}mix.left.{t}.b", (n,), "zero"))
                if a.get("conv"):
                    specs.append((f"{p}mix.left.{t}.conv", (n, a["conv"]), "w"))
            k, v = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            for t, shape, kind in (("q", (k, W), "w"), ("k", (k, W), "w"), ("v", (v, W), "w"), ("g", (v, W), "w"), ("o", (W, v), "w"), ("norm", (r["vdim"],), "one"), ("a1", (decay_rank, W), "w"), ("a2", (k, decay_rank), "w"), ("a2.b", (k,), "embed")):
                specs.append((f"{p}mix.right.{t}", shape, kind))
        else:
            h, d, r, rot = m["heads"], m["dim"], m["kv_rank"], m["rot_dim"]
            specs += [(p + "mix.dq", (m["q_rank"], W), "w"), (p + "mix.dq.norm", (m["q_rank"],), "one"), (p + "mix.uq", (h * (d + rot), m["q_rank"]), "w"), (p + "mix.dkv", (r + rot, W), "w"), (p + "mix.dkv.norm", (r,), "one")]
            specs += [(p + "mix.uk", (h * d, r), "w"), (p + "mix.uv", (h * m["vdim"], r), "w"), (p + "mix.o", (W, h * m["vdim"]), "w")]
        mlp = lambda q, ff: [(q + "gate", (ff, W), "w"), (q + "up", (ff, W), "w"), (q + "down", (W, ff), "w")]
        if f is None:
            continue
        if f["kind"] == "dense":
            specs += mlp(p + "mlp.", f["ff"])
        else:
            specs.append((p + "mlp.router", (f["router"]["experts"], W), "w"))
            for e in range(f["router"]["experts"]):
                specs += mlp(f"{p}mlp.e{e}.", f["expert"]["ff"])
            specs += mlp(p + "mlp.shared.", f["shared"]["ff"]) + [(p + "mlp.shared.sg", (1, W), "w")]
    return specs + [("final.norm", (W,), "zero")]


def gebilorn_tensor(seed: int, spec) -> np.ndarray:
    """bf16 bits of one tensor: linears N(0, 1/in), offsets and biases around 0, other vectors around 1."""
    name, shape, kind = spec
    if kind == "zero":
        return f32_to_bf16_rne(0.25 * _rng(seed, name).standard_normal(shape, dtype=np.float32))
    return tunitar_tensor(seed, spec)


def gebilorn_weights(cfg: dict, seed: int, decay_rank: int = 16) -> Dict[str, np.ndarray]:
    """name -> bf16 bits of every tensor."""
    return {s[0]: gebilorn_tensor(seed, s) for s in gebilorn_tensor_specs(cfg, decay_rank)}


def write_gebilorn_model(model_dir: str, cfg: dict, seed: int, weights: Optional[Dict[str, np.ndarray]] = None, decay_rank: int = 16) -> str:
    """config.json + model.safetensors of a Gebilorn model (weights: bits to write instead of the seeded ones)."""
    return _write_model(model_dir, cfg, gebilorn_tensor_specs(cfg, decay_rank), lambda s: gebilorn_tensor(seed, s) if weights is None else weights[s[0]])


# ---- Pulenex ----------------------------------------------------------------------------------


def pulenex_rot(dims: int, base: float = 10000.0) -> dict:
    return {"dims": dims, "base": base}


def pulenex_retention(heads: int, dim: int, vdim: int, rot: Optional[dict] = None, decay: Optional[List[float]] = None) -> dict:
    """decay: per head; by default heads that forget within 4, 8, 16, ... tokens, up to 2048."""
    decay = [1.0 - 2.0 ** -(2 + h % 10) for h in range(heads)] if decay is None else decay
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": rot or pulenex_rot(dim // 2 * 2), "decay": decay}}


def pulenex_parallel(left: Tuple[int, int, int], chunk: int, conv: int, right: Tuple[int, int, int, int], right_conv: int, rot: Optional[dict] = None, scale: Optional[float] = None) -> dict:
    """left: heads, kv_heads, dim of the chunked attention; right: heads, kv_heads, dim, vdim of the gated delta rule."""
    h, g, d = left
    a = {"heads": h, "kv_heads": g, "dim": d, "vdim": d, "scale": d**-0.5 if scale is None else scale, "mask": {"size": chunk}, "conv": conv, "rot": rot or pulenex_rot(d // 2 * 2)}
    return {"type": "parallel", "mixer": {"left": a, "right": dict(zip(("heads", "kv_heads", "dim", "vdim"), right), conv=right_conv)}}


def pulenex_latent(heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, window: int, kv_from: Optional[int] = None, base: float = 10000.0, scale: Optional[float] = None) -> dict:
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale, "mask": {"size": window}, "rot": pulenex_rot(rot_dim, base)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def pulenex_dense(ff: int, limit: float = 7.0) -> dict:
    return {"kind": "dense", "ff": ff, "limit": limit}


def pulenex_config(width: int, vocab: int, layers: List[Tuple[dict, Optional[dict]]], logit_scale: float = 1.0, eps: float = 1e-6, **extra) -> dict:
    """layers: (mixer, mlp or None) pairs."""
    return {"architecture": "Pulenex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": [{**m, "mlp": f} for m, f in layers], **extra}


def pulenex_uniform(width: int, vocab: int, n_layers: int, heads: int, kv_heads: int, dim: int, ff: int, kv_rank: int) -> dict:
    """Of every four layers one runs retention, one chunked attention beside the gated delta rule, two latent attention in a window, the
    second of which reads the first one's latents."""
    layers = []
    for i in range(n_layers):
        if i % 4 == 0:
            m = pulenex_retention(heads, dim, dim)
        elif i % 4 == 1:
            m = pulenex_parallel((heads, kv_heads, dim), 1024, 4, (heads, kv_heads, dim, dim), 4, pulenex_rot(dim, 500000.0))
        else:
            m = pulenex_latent(heads, dim, 64, dim, kv_rank, 1024, i - 1 if i % 4 == 3 else None)
        layers.append((m, pulenex_dense(ff)))
    return pulenex_config(width, vocab, layers)


# Pulenex stacks with the width, depth, heads, head size and MLP parameters of the Qwen2.5 architectures above.
PULENEX_05B = pulenex_uniform(896, 151936, 24, 14, 2, 64, 4864, 256)
PULENEX_15B = pulenex_uniform(1536, 151936, 28, 12, 2, 128, 8960, 512)


def pulenex_tensor_specs(cfg: dict, ranks: Tuple[int, int] = (64, 64)) -> List[Tuple[str, Tuple[int, ...], str]]:
    """(name, shape, kind); ranks: widths of the latents of decays and of output gates."""
    W, V = cfg["width"], cfg["vocab"]
    specs: List[Tuple[str, Tuple[int, ...], str]] = [("embed", (V, W), "embed")]
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        specs += [(p + "norm1", (W,), "one"), (p + "norm1b", (W,), "one")]
        if layer["type"] == "retention":
            k, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            specs += [(p + "mix.q", (k, W), "w"), (p + "mix.k", (k, W), "w"), (p + "mix.v", (v, W), "w"), (p + "mix.g", (v, W), "w"), (p + "mix.o", (W, v), "w")]
        elif layer["type"] == "parallel":
            a, r, l, t = m["left"], m["right"], p + "mix.left.", p + "mix.right."
            h, q, k = a["heads"], a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            specs += [(l + "q", (q, W), "w"), (l + "k", (k, W), "w"), (l + "q.conv", (q, a["conv"]), "tap"), (l + "k.conv", (k, a["conv"]), "tap"), (l + "talk", (h, h), "mix"), (l + "temp", (h,), "one"), (l + "sink", (h,), "embed")]
            specs += [(l + "g", (q, W), "w"), (l + "o", (W, q), "w"), (l + "out", (W,), "one")]
            h, k, v = r["heads"], r["kv_heads"] * r["dim"], r["heads"] * r["vdim"]
            specs += [(t + n, (c, W), "w") for n, c in (("q", k), ("k", k), ("v", v), ("b", h), ("a1", ranks[0]), ("g1", ranks[1]))] + [(t + n + ".conv", (c, r["conv"]), "tap") for n, c in (("q", k), ("k", k), ("v", v))]
            specs += [(t + "A_log", (h,), "rate"), (t + "a2", (h * r["dim"], ranks[0]), "w"), (t + "dt_bias", (h * r["dim"],), "embed"), (t + "g2", (v, ranks[1]), "w"), (t + "norm", (r["vdim"],), "one"), (t + "o", (W, v), "w"), (t + "out", (W,), "one")]
        else:
            h, d, r, rot = m["heads"], m["dim"], m["kv_rank"], m["rot_dim"]
            specs.append((p + "mix.q", (h * (d + rot), W), "w"))
            if m.get("kv_from") is None:
                specs += [(p + "mix.dkv", (r + rot, W), "w"), (p + "mix.dkv.norm", (r,), "one")]
            specs += [(p + "mix.uk", (h * d, r), "w"), (p + "mix.uv", (h * m["vdim"], r), "w"), (p + "mix.g", (h, W), "w"), (p + "mix.o", (W, h * m["vdim"]), "w")]
        if f is not None:
            ff = f["ff"]
            specs += [(p + "norm2", (W,), "one"), (p + "norm2b", (W,), "one"), (p + "mlp.gate", (ff, W), "w"), (p + "mlp.gate.b", (ff,), "zero"), (p + "mlp.up", (ff, W), "w"), (p + "mlp.up.b", (ff,), "zero")]
            specs += [(p + "mlp.down", (W, ff), "w"), (p + "mlp.down.b", (W,), "zero")]
    return specs + [("final.norm", (W,), "one"), ("head", (V, W), "w")]


def pulenex_tensor(seed: int, spec) -> np.ndarray:
    """bf16 bits of one tensor: linears N(0, 1/in), biases around 0, mixing matrices around the identity, decay rates from 1/16 to 1, other
    vectors around 1."""
    name, shape, kind = spec
    g = _rng(seed, name)
    if kind == "tap":
        return f32_to_bf16_rne(float(shape[1]) ** -0.5 * g.standard_normal(shape, dtype=np.float32))
    if kind == "mix":
        return f32_to_bf16_rne((np.eye(shape[0]) + 0.3 * g.standard_normal(shape, dtype=np.float32)).astype(np.float32))
    if kind == "rate":
        return f32_to_bf16_rne(np.log(2.0 ** (-4.0 * g.random(shape, dtype=np.float32))).astype(np.float32))
    return gebilorn_tensor(seed, spec)


def pulenex_weights(cfg: dict, seed: int, ranks: Tuple[int, int] = (64, 64)) -> Dict[str, np.ndarray]:
    """name -> bf16 bits of every tensor."""
    return {s[0]: pulenex_tensor(seed, s) for s in pulenex_tensor_specs(cfg, ranks)}


def write_pulenex_model(model_dir: str, cfg: dict, seed: int, weights: Optional[Dict[str, np.ndarray]] = None, ranks: Tuple[int, int] = (64, 64)) -> str:
    """config.json + model.safetensors of a Pulenex model (weights: bits to write instead of the seeded ones)."""
    return _write_model(model_dir, cfg, pulenex_tensor_specs(cfg, ranks), lambda s: pulenex_tensor(seed, s) if weights is None else weights[s[0]])


def shard_hf_model(src_dir: str, dst_dir: str, n_shards: int = 2) -> str:
    """Rewrite a single-file checkpoint as `n_shards` safetensors files plus model.safetensors.index.json,
    the layout HfModel::load_with_dtype falls back to (src/hf/model.rs:86-127).  Tensors are dealt out
    round-robin, so every shard holds pieces of every layer."""
    os.makedirs(dst_dir, exist_ok=True)
    with open(os.path.join(src_dir, "config.json")) as f, open(os.path.join(dst_dir, "config.json"), "w") as g:
        g.write(f.read())
    tensors = read_safetensors(os.path.join(src_dir, "model.safetensors"))
    names = list(tensors)
    weight_map = {}
    for sh in range(n_shards):
        fname = f"model-{sh + 1:05d}-of-{n_shards:05d}.safetensors"
        mine = names[sh::n_shards]
        header, off = {}, 0
        for name in mine:
            dt, shape, arr = tensors[name]
            header[name] = {"dtype": dt, "shape": list(shape), "data_offsets": [off, off + arr.nbytes]}
            off += arr.nbytes
            weight_map[name] = fname
        hjson = json.dumps(header, separators=(",", ":")).encode()
        hjson += b" " * ((8 - len(hjson) % 8) % 8)
        with open(os.path.join(dst_dir, fname), "wb") as f:
            f.write(struct.pack("<Q", len(hjson)))
            f.write(hjson)
            for name in mine:
                f.write(np.ascontiguousarray(tensors[name][2]).tobytes())
    with open(os.path.join(dst_dir, "model.safetensors.index.json"), "w") as f:
        json.dump({"metadata": {"total_size": sum(t[2].nbytes for t in tensors.values())}, "weight_map": weight_map}, f)
    return dst_dir


def read_safetensors(path: str) -> Dict[str, Tuple[str, Tuple[int, ...], np.ndarray]]:
    """name -> (dtype string, shape, raw array view).  BF16/F16 come back as uint16 bits."""
    raw = np.memmap(path, dtype=np.uint8, mode="r")
    (hlen,) = struct.unpack("<Q", raw[:8].tobytes())
    header = json.loads(raw[8 : 8 + hlen].tobytes())
    base = 8 + hlen
    np_of = {"BF16": np.uint16, "F16": np.uint16, "F32": np.float32, "F64": np.float64, "I32": np.int32, "I64": np.int64}
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        b, e = info["data_offsets"]
        arr = raw[base + b : base + e].view(np_of[info["dtype"]]).reshape(info["shape"])
        out[name] = (info["dtype"], tuple(info["shape"]), arr)
    return out


# ----------------------------------------------------------------------------------------
# GGUF
# ----------------------------------------------------------------------------------------


def quant_blocks(seed: int, name: str, n_out: int, n_in: int, ggml_type: int) -> np.ndarray:
    """Random blocks [n_out, n_in/32] in GGUF byte order: f16 scale |N(0,0.01)| + codes
    (Q8_0 / Q4_0), or super-blocks [n_out, n_in/256] of 144 (Q4_K) / 210 (Q6_K) bytes."""
    assert n_in % 32 == 0
    g = _rng(seed, name)
    if ggml_type in (GGML_Q4_K, GGML_Q6_K):
        assert n_in % 256 == 0, "K-quants need in_features to be a multiple of 256"
        nsb = n_out * (n_in // 256)
        if ggml_type == GGML_Q4_K:
            blk = g.integers(0, 256, size=(nsb, 144), dtype=np.uint8)  # packed 6-bit scales/mins and nibbles: any byte is valid
            d = np.abs(g.standard_normal(nsb, dtype=np.float32) * np.float32(4e-4)).astype(np.float16)
            dmin = np.abs(g.standard_normal(nsb, dtype=np.float32) * np.float32(1e-4)).astype(np.float16)
            blk[:, 0:2] = d.view(np.uint8).reshape(nsb, 2)
            blk[:, 2:4] = dmin.view(np.uint8).reshape(nsb, 2)
        else:
            blk = g.integers(0, 256, size=(nsb, 210), dtype=np.uint8)
            blk[:, 192:208] = g.integers(-64, 64, size=(nsb, 16), dtype=np.int8).view(np.uint8)  # i8 sub-block scales
            d = np.abs(g.standard_normal(nsb, dtype=np.float32) * np.float32(2e-5)).astype(np.float16)
            blk[:, 208:210] = d.view(np.uint8).reshape(nsb, 2)
        return blk.reshape(-1)
    nb = n_out * (n_in // 32)
    scale = np.abs(g.standard_normal(nb, dtype=np.float32) * np.float32(0.01)).astype(np.float16)
    if ggml_type == GGML_Q8_0:
        codes = g.integers(-127, 128, size=(nb, 32), dtype=np.int8).view(np.uint8)
        blk = np.empty((nb, 34), dtype=np.uint8)
    elif ggml_type == GGML_Q4_0:
        nib = g.integers(0, 16, size=(nb, 32), dtype=np.uint8)
        codes = (nib[:, :16] | (nib[:, 16:] << 4)).astype(np.uint8)
        blk = np.empty((nb, 18), dtype=np.uint8)
    else:
        raise ValueError(ggml_type)
    blk[:, 0:2] = scale.view(np.uint8).reshape(nb, 2)
    blk[:, 2:] = codes
    return blk.reshape(-1)


def _gguf_str(s: str) -> bytes:
    b = s.encode()
    return struct.pack("<Q", len(b)) + b


def _gguf_kv(key: str, val) -> bytes:
    out = _gguf_str(key)
    if isinstance(val, str):
        out += struct.pack("<I", 8) + _gguf_str(val)
    elif isinstance(val, bool):
        out += struct.pack("<IB", 7, int(val))
    elif isinstance(val, float):
        out += struct.pack("<If", 6, val)
    elif isinstance(val, int):
        out += struct.pack("<II", 4, val)
    else:
        raise TypeError(type(val))
    return out


def write_gguf(path: str, metadata: Dict[str, object], tensors: Iterable[Tuple[str, Tuple[int, ...], int, np.ndarray]], alignment: int = 32) -> None:
    """tensors: (name, logical shape outermost-first, ggml type, raw bytes as uint8/uint16 array)."""
    tensors = list(tensors)
    head = struct.pack("<IIQQ", GGUF_MAGIC, 3, len(tensors), len(metadata))
    for k, v in metadata.items():
        head += _gguf_kv(k, v)
    infos = b""
    off = 0
    offsets = []
    for name, shape, gt, data in tensors:
        nbytes = data.nbytes
        infos += _gguf_str(name) + struct.pack("<I", len(shape))
        for d in reversed(shape):  # GGUF stores dims innermost-first (src/gguf.rs:412-417)
            infos += struct.pack("<Q", d)
        infos += struct.pack("<IQ", gt, off)
        offsets.append(off)
        off += (nbytes + alignment - 1) // alignment * alignment
    pre = head + infos
    pad = (alignment - len(pre) % alignment) % alignment
    with open(path, "wb") as f:
        f.write(pre + b"\0" * pad)
        for (name, shape, gt, data), o in zip(tensors, offsets):
            b = data.tobytes()
            f.write(b)
            f.write(b"\0" * ((alignment - len(b) % alignment) % alignment))


def gguf_metadata(cfg: DecoderConfig, arch: str = "llama") -> Dict[str, object]:
    md: Dict[str, object] = {
        "general.architecture": arch,
        f"{arch}.embedding_length": cfg.hidden_size,
        f"{arch}.feed_forward_length": cfg.intermediate_size,
        f"{arch}.attention.head_count": cfg.num_attention_heads,
        f"{arch}.block_count": cfg.num_hidden_layers,
        f"{arch}.attention.head_count_kv": cfg.num_key_value_heads,
        f"{arch}.vocab_size": cfg.vocab_size,
        f"{arch}.attention.layer_norm_rms_epsilon": float(cfg.rms_norm_eps),
        f"{arch}.rope.freq_base": float(cfg.rope_theta),
        f"{arch}.context_length": cfg.max_position_embeddings,
    }
    if cfg.head_dim is not None:
        md[f"{arch}.attention.key_length"] = cfg.head_dim
    return md


def write_gguf_model(path: str, cfg: DecoderConfig, seed: int, ggml_type: int, quant_lm_head: bool = True, norm_jitter: float = 0.0, k_mix: bool = False, quant_embed: bool = False) -> str:
    """GGUF file: all linears in ``ggml_type`` blocks, bf16 embedding/norms, optional biases (f32).
    ``k_mix`` writes attn_v, ffn_down and output as Q6_K beside Q4_K elsewhere (the mix of a Q4_K_M
    file); ``quant_embed`` quantises token_embd too (Q6_K, or ``ggml_type`` for the 32-value formats)."""
    H, I, V = cfg.hidden_size, cfg.intermediate_size, cfg.vocab_size
    q6_names = ("attn_v.weight", "ffn_down.weight", "output.weight") if k_mix else ()

    def norm(name, n):
        if norm_jitter > 0:
            v = 1.0 + norm_jitter * _rng(seed, name).standard_normal(n, dtype=np.float32)
            return (name, (n,), GGML_BF16, f32_to_bf16_rne(v))
        return (name, (n,), GGML_BF16, ones_bf16((n,)))

    def lin(name, out_f, in_f):
        gt = GGML_Q6_K if name.endswith(q6_names) and q6_names else ggml_type
        return (name, (out_f, in_f), gt, quant_blocks(seed, name, out_f, in_f, gt))

    def gen():
        if quant_embed:
            gt = GGML_Q6_K if ggml_type in (GGML_Q4_K, GGML_Q6_K) else ggml_type
            yield ("token_embd.weight", (V, H), gt, quant_blocks(seed, "token_embd.weight", V, H, gt))
        else:
            yield ("token_embd.weight", (V, H), GGML_BF16, normal_bf16(seed, "token_embd.weight", (V, H)))
        for i in range(cfg.num_hidden_layers):
            p = f"blk.{i}."
            yield norm(p + "attn_norm.weight", H)
            for nm, out_f in (("q", cfg.q_dim), ("k", cfg.kv_dim), ("v", cfg.kv_dim)):
                yield lin(p + f"attn_{nm}.weight", out_f, H)
                if cfg.qkv_bias:
                    b = _rng(seed, p + f"attn_{nm}.bias").standard_normal(out_f, dtype=np.float32) * np.float32(0.02)
                    yield (p + f"attn_{nm}.bias", (out_f,), GGML_F32, b)
            if cfg.qk_norm:
                yield norm(p + "attn_q_norm.weight", cfg.hd)
                yield norm(p + "attn_k_norm.weight", cfg.hd)
            yield lin(p + "attn_output.weight", H, cfg.q_dim)
            yield norm(p + "ffn_norm.weight", H)
            yield lin(p + "ffn_gate.weight", I, H)
            yield lin(p + "ffn_up.weight", I, H)
            yield lin(p + "ffn_down.weight", H, I)
        yield norm("output_norm.weight", H)
        if not cfg.tie_word_embeddings:
            if quant_lm_head:
                yield lin("output.weight", V, H)
            else:
                yield ("output.weight", (V, H), GGML_BF16, normal_bf16(seed, "output.weight", (V, H)))

    write_gguf(path, gguf_metadata(cfg), gen())
    return path


def read_gguf(path: str):
    """Minimal GGUF v2/v3 reader: returns (metadata dict, {name: (shape, ggml_type, uint8 view)})."""
    raw = np.memmap(path, dtype=np.uint8, mode="r")
    pos = 0

    def rd(fmt):
        nonlocal pos
        sz = struct.calcsize(fmt)
        v = struct.unpack("<" + fmt, raw[pos : pos + sz].tobytes())
        pos += sz
        return v if len(v) > 1 else v[0]

    def rstr():
        nonlocal pos
        n = rd("Q")
        s = raw[pos : pos + n].tobytes().decode()
        pos += n
        return s

    magic, version = rd("II")
    assert magic == GGUF_MAGIC and version in (2, 3)
    nt, nkv = (rd("QQ") if version >= 3 else rd("II"))
    scalar = {0: "B", 1: "b", 2: "H", 3: "h", 4: "I", 5: "i", 6: "f", 7: "B", 10: "Q", 11: "q", 12: "d"}

    def rval(t):
        if t == 8:
            return rstr()
        if t == 9:
            et = rd("I")
            n = rd("Q")
            return [rval(et) for _ in range(n)]
        v = rd(scalar[t])
        return bool(v) if t == 7 else v

    md = {}
    for _ in range(nkv):
        k = rstr()
        t = rd("I")
        md[k] = rval(t)
    align = int(md.get("general.alignment", 32))
    infos = []
    for _ in range(nt):
        name = rstr()
        nd = rd("I")
        dims = [rd("Q") for _ in range(nd)]
        dims.reverse()
        gt = rd("I")
        off = rd("Q")
        infos.append((name, tuple(dims), gt, off))
    data0 = (pos + align - 1) // align * align
    bpe = {GGML_F32: (1, 4), GGML_F16: (1, 2), GGML_BF16: (1, 2), GGML_Q8_0: (32, 34), GGML_Q4_0: (32, 18), GGML_Q4_K: (256, 144), GGML_Q6_K: (256, 210)}
    tensors = {}
    for name, shape, gt, off in infos:
        bs, ts = bpe[gt]
        nbytes = int(np.prod(shape)) // bs * ts
        tensors[name] = (shape, gt, raw[data0 + off : data0 + off + nbytes])
    return md, tensors


def prompt_ids(seed: int, n: int, vocab: int) -> np.ndarray:
    """Prompt token ids uniform in [0, vocab)."""
    return _rng(seed, "prompt").integers(0, vocab, size=n, dtype=np.int64)
