"""Seeded synthetic inputs with the benchmark's shapes and value distributions.

They stand in for real Qwen3 weights (not available offline).  Host versions
(numpy, PCG64) feed both the oracle and the device path in the parity tests; the
``*_device`` versions fill large benchmark buffers directly in HBM with torch's
generator.

Distributions: weights are int4 symmetric integers uniform in [-7, 7] stored as
offset-binary nibbles (q + 8), two per byte along K, even k in the low nibble;
one binary16 scale per 16-element k-block drawn as |N(0, 0.02)| + 1e-3 (the fp32
copy used by the reference-format path is the same value widened);
activations are binary16 N(0, 1); norm weights 1 + 0.1 N(0, 1).
"""
from __future__ import annotations

import numpy as np

SEED_BASE = 0xB2000000


def rng(seed: int) -> np.random.Generator:
    return np.random.Generator(np.random.PCG64(SEED_BASE + int(seed)))


def int4_weights(N: int, K: int, seed: int, full_range: bool = False):
    """-> (W_packed u8 [N][K/2], scale_f16 [N][K/16], scale_f32 [N][K/16]).
    ``full_range`` also emits nibble 0 (q = -8), which real weight files never
    hold but the kernels must decode."""
    g = rng(seed)
    lo, hi = (-8, 8) if full_range else (-7, 8)
    q = g.integers(lo, hi, size=(N, K), dtype=np.int8)
    nib = (q + 8).astype(np.uint8)
    packed = (nib[:, 0::2] | (nib[:, 1::2] << 4)).astype(np.uint8)
    sc = (np.abs(g.normal(0.0, 0.02, size=(N, K // 16))) + 1e-3).astype(np.float16)
    return np.ascontiguousarray(packed), sc, sc.astype(np.float32)


def activations_f16(M: int, K: int, seed: int) -> np.ndarray:
    return rng(seed).normal(0.0, 1.0, size=(M, K)).astype(np.float16)


def norm_weight(H: int, seed: int) -> np.ndarray:
    return (1.0 + 0.1 * rng(seed).normal(0.0, 1.0, size=H)).astype(np.float32)


def kv_cache_f16(shape, seed: int) -> np.ndarray:
    return rng(seed).normal(0.0, 1.0, size=shape).astype(np.float16)


# ---------------------------------------------------------------- device side
def int4_weights_device(N: int, K: int, seed: int, device="cuda", scale_dtype=None):
    """Same distributions, generated in HBM: (W_packed u8, scale f16 or f32)."""
    import torch

    gen = torch.Generator(device=device)
    gen.manual_seed(SEED_BASE + int(seed))
    lo = torch.randint(1, 16, (N, K // 2), dtype=torch.uint8, device=device, generator=gen)
    hi = torch.randint(1, 16, (N, K // 2), dtype=torch.uint8, device=device, generator=gen)
    packed = lo | (hi << 4)
    del lo, hi
    sc = torch.empty((N, K // 16), dtype=torch.float32, device=device)
    sc.normal_(0.0, 0.02, generator=gen)
    sc = sc.abs_().add_(1e-3).to(torch.float16)
    if scale_dtype is not None and scale_dtype != torch.float16:
        sc = sc.to(scale_dtype)
    return packed, sc


def activations_f16_device(M: int, K: int, seed: int, device="cuda"):
    import torch

    gen = torch.Generator(device=device)
    gen.manual_seed(SEED_BASE + int(seed))
    x = torch.empty((M, K), dtype=torch.float32, device=device)
    x.normal_(0.0, 1.0, generator=gen)
    return x.to(torch.float16)


def write_random_model(directory: str, cfg: dict, seed: int = 0, device="cuda") -> int:
    """A config.json model with random bfloat16 weights (values scaled by fan-in); returns the bytes of its matrices."""
    import json
    import os
    import struct

    import torch

    W, V = cfg["width"], cfg["vocab"]
    shapes = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q, H, vd = p + "mix.", m["heads"], m["vdim"]
        shapes[p + "norm1"] = (W,)
        if cfg["architecture"] == "Lanedra":
            shapes[p + "norm1b"] = (W,)
            if L["mlp"]:
                shapes[p + "norm2b"] = (W,)
        if L["type"] == "delta":
            D, G = m["dim"], m["kv_heads"]
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * vd)):
                shapes.update({q + n: (rows, W), q + n + ".conv": (rows, m["conv"])})
            shapes.update({q + "a": (H, W), q + "b": (H, W), q + "g": (H * vd, W), q + "A_log": (H,), q + "dt_bias": (H,), q + "norm": (vd,)})
        elif L["type"] == "attention":
            D, G = m["dim"], m["kv_heads"]
            shapes[q + "q"] = (H * 2 * D, W)
            if "kv_from" not in m:
                shapes.update({q + "k": (G * 2 * D, W), q + "v": (G * vd, W)})
            shapes.update({q + n: (D,) for n in ("lq1", "lk1", "lq2", "lk2")})
        elif L["type"] == "mamba2":
            inner, gn = H * vd, m["groups"] * m["state"]
            shapes.update({q + "in": (2 * inner + 2 * gn + H, W), q + "conv": (inner + 2 * gn, m["conv"]), q + "conv.b": (inner + 2 * gn,),
                           q + "dt_bias": (H,), q + "A_log": (H,), q + "D": (H,), q + "norm": (inner,)})
        elif L["type"] == "retention":
            shapes.update({q + "q": (H * m["dim"], W), q + "k": (H * m["dim"], W), q + "v": (H * vd, W), q + "g": (H * vd, W)})
        else:
            R, rot = m["kv_rank"], m["rot_dim"]
            shapes.update({q + "q": (H * (m["dim"] + rot), W), q + "uk": (H * m["dim"], R), q + "uv": (H * vd, R), q + "sink": (H,),
                           q + "g": (H, W)})
            if "kv_from" not in m:
                shapes.update({q + "dkv": (R + rot, W), q + "dkv.norm": (R,)})
        shapes[q + "o"] = (W, H * vd)
        if L["mlp"]:
            ff = L["mlp"]["ff"]
            shapes.update({p + "norm2": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    header, at, matrices = {}, 0, 0
    for name, shape in shapes.items():
        n = 2 * int(np.prod(shape))
        header[name] = {"dtype": "BF16", "shape": list(shape), "data_offsets": [at, at + n]}
        at += n
        if len(shape) == 2 and not name.endswith(".conv") and name != "embed":
            matrices += n
    gen = torch.Generator(device=device).manual_seed(seed)
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(os.path.join(directory, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for name, shape in shapes.items():
            t = torch.randn(shape, generator=gen, device=device)
            if len(shape) == 2 and name != "embed":
                t *= shape[1] ** -0.5
            elif name.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b")):
                around_zero = cfg["architecture"] == "Lanedra" and not name.endswith("mix.norm")
                t = (0.0 if around_zero else 1.0) + 0.1 * t
            elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
                t *= 0.1
            elif name.endswith("dt_bias"):
                t = t - 4.0
            f.write(t.to(torch.bfloat16).view(torch.int16).cpu().numpy().tobytes())
    return matrices
