"""Small random config.json models for the tests: configurations, weights, the directory a model is loaded from, and the
float64 answer of oracle.lm_layers.  Weights are rounded to bfloat16 first, so that every side sees the same values."""
import copy
import json
import os
import struct

import numpy as np

from oracle import lm_layers as plain


def to_bf16(a):
    """float -> (bfloat16 bits, the rounded values)"""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    bits = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)
    return bits, (bits.astype(np.uint32) << 16).view(np.float32).astype(np.float64)


def mamba2(heads, vdim, state, groups, conv, norm_groups):
    return "mamba2", dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)


def retention(heads, dim, vdim, decay):
    assert len(decay) == heads
    return "retention", dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay))


def latent(heads, dim, rot, rank, vdim, scale, base=10000.0, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot, kv_rank=rank, vdim=vdim, scale=scale, rot=dict(base=base, dims=rot))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "latent_attention", m


def delta(heads, kv_heads, dim, vdim, conv):
    return "delta", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


def yarn(factor, original, fast=32.0, slow=1.0):
    return dict(factor=factor, original=original, fast=fast, slow=slow)


def diff_attention(heads, kv_heads, dim, vdim, window, rot_dims=None, base=10000.0, scaling=None, diff=0.4, scale=None, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=window), diff=diff,
             scale=1.3 * dim ** -0.5 if scale is None else scale, rot=dict(base=base, dims=dim // 2 * 2 if rot_dims is None else rot_dims))
    if scaling is not None:
        m["rot"]["scaling"] = scaling
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention", m


def _layers(layers, ff):
    return [{"type": t, "mixer": copy.deepcopy(m), "mlp": None if f is None else {"kind": "dense", "ff": f}}
            for (t, m), f in zip(layers, ff)]


def config(width, vocab, layers, ff, eps=1e-5, softcap=20.0):
    """layers: list of (type, mixer); ff: one size per layer, None for no feed-forward."""
    return {"architecture": "Vifivik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": softcap,
            "layers": _layers(layers, ff)}


def lanedra(width, vocab, layers, ff, eps=1e-5, scale=1.7):
    return {"architecture": "Lanedra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": _layers(layers, ff)}


def lanedra_tensors(cfg, seed):
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]

    def mat(n, k, gain=1.0):
        return rng.standard_normal((n, k)) * gain / np.sqrt(k)

    def offsets(n, mean=0.0):
        return mean + rng.uniform(-0.3, 0.3, n)

    w = {"embed": rng.standard_normal((V, W)), "head": mat(V, W, 3.0), "final.norm": offsets(W)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        H, G, D, Vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w[p + "norm1"], w[p + "norm1b"] = offsets(W), offsets(W, -0.2)
        if L["type"] == "delta":
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * Vd)):
                w[q + n] = mat(rows, W)
                w[q + n + ".conv"] = rng.standard_normal((rows, m["conv"])) * 0.6
            w[q + "b"], w[q + "a"], w[q + "g"] = mat(H, W, 2.0), mat(H, W), mat(H * Vd, W)
            w[q + "A_log"], w[q + "dt_bias"] = np.log(rng.uniform(0.5, 8.0, H)), rng.uniform(-5.0, 0.0, H)
            w[q + "norm"] = rng.uniform(0.6, 1.4, Vd)
        else:
            w[q + "q"] = mat(H * 2 * D, W, 1.5)
            if "kv_from" not in m:
                w[q + "k"], w[q + "v"] = mat(G * 2 * D, W, 1.5), mat(G * Vd, W)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[q + n] = rng.standard_normal(D) * 0.6 * D ** -0.25
        w[q + "o"] = mat(W, H * Vd)
        if L["mlp"] is not None:
            w[p + "norm2"], w[p + "norm2b"] = offsets(W), offsets(W, -0.2)
            w[p + "mlp.gate"], w[p + "mlp.up"] = mat(L["mlp"]["ff"], W), mat(L["mlp"]["ff"], W)
            w[p + "mlp.down"] = mat(W, L["mlp"]["ff"])
    return w


def tensors(cfg, seed):
    if cfg["architecture"] == "Lanedra":
        return lanedra_tensors(cfg, seed)
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]

    def mat(n, k, gain=1.0):
        return rng.standard_normal((n, k)) * gain / np.sqrt(k)

    def gains(n, lo=0.6, hi=1.4):
        return rng.uniform(lo, hi, n)

    w = {"embed": rng.standard_normal((V, W)), "head": mat(V, W, 6.0), "final.norm": gains(W)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        H, Vd = m["heads"], m["vdim"]
        w[p + "norm1"] = gains(W, 0.3, 0.8)
        if L["type"] == "mamba2":
            inner, gn = H * Vd, m["groups"] * m["state"]
            w[q + "in"] = mat(2 * inner + 2 * gn + H, W)
            w[q + "conv"] = rng.standard_normal((inner + 2 * gn, m["conv"])) * 0.5
            w[q + "conv.b"] = rng.standard_normal(inner + 2 * gn) * 0.2
            w[q + "dt_bias"] = rng.uniform(-5.0, 0.0, H)
            w[q + "A_log"] = np.log(rng.uniform(0.5, 8.0, H))
            w[q + "D"] = rng.standard_normal(H)
            w[q + "norm"] = gains(inner)
        elif L["type"] == "retention":
            for n, rows in (("q", H * m["dim"]), ("k", H * m["dim"]), ("v", H * Vd), ("g", H * Vd)):
                w[q + n] = mat(rows, W)
        else:
            w[q + "q"] = mat(H * (m["dim"] + m["rot_dim"]), W)
            if "kv_from" not in m:
                w[q + "dkv"] = mat(m["kv_rank"] + m["rot_dim"], W)
                w[q + "dkv.norm"] = gains(m["kv_rank"])
            w[q + "uk"] = mat(H * m["dim"], m["kv_rank"])
            w[q + "uv"] = mat(H * Vd, m["kv_rank"])
            w[q + "sink"] = rng.uniform(-1.0, 3.0, H)
            w[q + "g"] = mat(H, W)
        w[q + "o"] = mat(W, H * Vd)
        if L["mlp"] is not None:
            w[p + "norm2"] = gains(W, 0.3, 0.8)
            w[p + "mlp.gate"], w[p + "mlp.up"] = mat(L["mlp"]["ff"], W), mat(L["mlp"]["ff"], W)
            w[p + "mlp.down"] = mat(W, L["mlp"]["ff"])
    return w


class Model:
    """A model directory and its plain evaluation."""

    def __init__(self, root, cfg, seed=0, weights=None):
        self.dir, self.cfg = str(root), cfg
        os.makedirs(self.dir, exist_ok=True)
        raw = tensors(cfg, seed) if weights is None else weights
        self.w, header, blobs, at = {}, {}, [], 0
        for name, a in raw.items():
            bits, self.w[name] = to_bf16(a)
            self.w[name] = self.w[name].reshape(np.shape(a))
            header[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [at, at + 2 * bits.size]}
            at += 2 * bits.size
            blobs.append(bits.tobytes())
        head = json.dumps(header).encode()
        with open(os.path.join(self.dir, "model.safetensors"), "wb") as f:
            f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
        with open(os.path.join(self.dir, "config.json"), "w") as f:
            json.dump(cfg, f)

    def plain(self, tokens):
        return plain.forward(self.cfg, self.w, tokens)

    def bar(self, tokens, f32):
        """Largest error a test accepts: a few times what rounding the inputs and outputs of every product and the outputs of
        silu to bfloat16 does to the logits of these tokens; for the 32-bit mode the same amplification applied to fp32
        roundings, whose sum over a row grows with the row's length."""
        def rounded(x):
            return to_bf16(x)[1].reshape(np.shape(x))

        def product(W, x):
            y = linear(W, rounded(x))
            return y if len(W) == self.cfg["vocab"] else rounded(y)

        exact = self.plain(tokens)[0]
        linear, silu = plain.linear, plain.silu
        try:
            plain.linear, plain.silu = product, lambda z: rounded(silu(z))
            noise = rel_error(self.plain(tokens)[0], exact).max()
        finally:
            plain.linear, plain.silu = linear, silu
        return 4 * noise * (2.0 ** -13 * max(1.0, self.cfg["width"] / 512) ** 0.5 if f32 else 1.0)

    def greedy(self, prompt, n):
        seq = list(prompt)
        for _ in range(n):
            seq.append(int(np.argmax(self.plain(seq)[0][-1])))
        return seq[len(prompt):]


def rel_error(got, want):
    """Per position: root mean square of the difference (mean taken off) over that of the wanted logits."""
    d = np.asarray(got, np.float64) - want
    d = d - d.mean(-1, keepdims=True)
    scale = np.sqrt(np.mean(np.square(want - want.mean(-1, keepdims=True))))
    return np.sqrt(np.mean(d * d, -1)) / scale


SINGLE = {   # one mixer each, sizes that are not multiples of anything
    "mamba2": lambda: config(60, 83, [mamba2(6, 20, 28, 3, 4, 5)], [None]),
    "mamba2_one_group": lambda: config(52, 64, [mamba2(5, 33, 12, 1, 2, 1)], [36], eps=1e-3),
    "mamba2_no_window": lambda: config(40, 50, [mamba2(2, 16, 70, 2, 1, 2)], [None]),
    "mamba2_wide_state": lambda: config(64, 70, [mamba2(2, 72, 200, 1, 3, 4)], [None]),
    "retention": lambda: config(44, 71, [retention(3, 20, 36, [0.9, 0.99, 0.999])], [None]),
    "retention_edges": lambda: config(48, 64, [retention(4, 136, 8, [0.0, 1.0, 0.5, 0.96875])], [28]),
    "mamba2_many_heads": lambda: config(48, 64, [mamba2(76, 40, 136, 4, 4, 19)], [None]),
    "retention_many_heads": lambda: config(48, 64, [retention(80, 20, 40, list(np.linspace(0.5, 1.0, 80)))], [None]),
    "latent": lambda: config(56, 79, [latent(3, 12, 6, 36, 20, 0.25)], [None]),
    "latent_many_heads": lambda: config(72, 90, [latent(21, 8, 4, 24, 12, 0.3, base=500.0)], [40]),
    "latent_wide_values": lambda: config(64, 64, [latent(2, 40, 24, 264, 150, 0.12)], [None]),
    "latent_long_rank": lambda: config(48, 64, [latent(17, 24, 8, 576, 72, 0.2)], [None]),
    "latent_very_long_rank": lambda: config(48, 64, [latent(2, 16, 8, 1100, 24, 0.2)], [None]),
}


def mixed():
    """Every mechanism together: order of layers, shared caches with other head counts, layers without feed-forward."""
    return config(88, 131, [
        latent(5, 20, 8, 44, 28, 0.21),
        mamba2(4, 24, 20, 2, 4, 8),
        latent(3, 36, 8, 44, 12, 0.4, kv_from=0),
        retention(2, 28, 44, [0.96875, 0.998046875]),
        mamba2(3, 40, 36, 1, 3, 1),
        latent(18, 12, 10, 100, 20, 0.3, base=777.0),
        latent(2, 44, 8, 44, 60, 0.15, kv_from=0),
        retention(5, 12, 20, [0.5, 0.9, 0.99, 0.999, 1.0])],
        [52, None, 40, 68, None, 33, None, 24], eps=2e-6, softcap=15.0)


KEY, QUERY = 1, 2   # tokens of needle_model


def needle_model(root, rank=40, heads=3):
    """One latent-attention layer in which token QUERY attends to token KEY with a score far above all others, wherever
    KEY stands."""
    cfg = config(64, 60, [latent(heads, 16, 8, rank, 24, 0.25)], [None])
    w = tensors(cfg, 77)
    w["l0.norm1"] = w["l0.norm1"] * 4.0
    m = cfg["layers"][0]["mixer"]
    c = plain.rms_norm(w["l0.mix.dkv"][:m["kv_rank"]] @ w["embed"][KEY], w["l0.mix.dkv.norm"], cfg["norm"]["eps"])
    key = (w["l0.mix.uk"] @ c).reshape(heads, m["dim"])
    e = w["embed"][QUERY]
    q = w["l0.mix.q"].reshape(heads, m["dim"] + m["rot_dim"], -1)
    for h in range(heads):
        q[h, :m["dim"]] += np.outer(key[h] * (40.0 / m["scale"] / (key[h] @ key[h])), e / (e @ e))
    return Model(root, cfg, weights=w)


def needle_tokens(length, key_at, query_at, seed=0):
    tok = np.random.default_rng(seed).integers(3, 60, length)
    tok[list(np.atleast_1d(key_at))] = KEY
    tok[list(np.atleast_1d(query_at))] = QUERY
    return tok


# ------------------------------------------------------------------------------------------- Lanedra
LANEDRA = {   # one mixer each
    "delta": lambda: lanedra(60, 83, [delta(6, 3, 20, 28, 4)], [None]),
    "delta_no_window": lambda: lanedra(52, 64, [delta(5, 1, 33, 12, 1)], [36], eps=1e-3, scale=0.4),
    "delta_own_keys": lambda: lanedra(40, 50, [delta(4, 4, 72, 40, 2)], [None]),
    "delta_wide_state": lambda: lanedra(64, 70, [delta(4, 2, 200, 72, 3)], [None]),
    "delta_very_wide_state": lambda: lanedra(64, 70, [delta(2, 1, 300, 33, 3)], [None]),
    "delta_many_heads": lambda: lanedra(48, 64, [delta(80, 16, 24, 40, 7)], [None]),
    "delta_many_wide_heads": lambda: lanedra(48, 64, [delta(78, 39, 136, 36, 2)], [None]),
    "diff": lambda: lanedra(56, 79, [diff_attention(6, 3, 12, 20, 9)], [None]),
    "diff_itself_only": lambda: lanedra(44, 60, [diff_attention(3, 1, 16, 24, 1, rot_dims=8)], [28]),
    "diff_whole_context": lambda: lanedra(48, 64, [diff_attention(4, 4, 20, 36, 100000, rot_dims=0, diff=0.0)], [None]),
    "diff_scaled_rotation": lambda: lanedra(72, 90, [diff_attention(4, 2, 24, 32, 64, base=700.0, scaling=yarn(6.0, 48, 5.0, 0.4))], [40], scale=1.0),
    "diff_partly_rotated": lambda: lanedra(72, 90, [diff_attention(4, 2, 40, 24, 33, rot_dims=16, base=50.0, scaling=yarn(3.0, 64))], [None], eps=1e-2),
    "diff_two_head_tiles": lambda: lanedra(64, 64, [diff_attention(20, 2, 9, 13, 50, rot_dims=6, diff=0.6)], [None]),
    "diff_mid": lambda: lanedra(48, 64, [diff_attention(3, 1, 100, 92, 70)], [None]),
    "diff_wide": lambda: lanedra(48, 64, [diff_attention(2, 1, 72, 150, 40, rot_dims=32)], [None]),
    "diff_very_wide": lambda: lanedra(48, 64, [diff_attention(2, 2, 40, 264, 45)], [None]),
    "odd_width": lambda: lanedra(46, 51, [delta(3, 1, 10, 14, 3)], [27]),
    "odd_wide_width": lambda: lanedra(2101, 40, [diff_attention(2, 1, 16, 20, 30)], [24]),
    "wide_width": lambda: lanedra(8452, 40, [delta(2, 1, 16, 20, 3)], [24]),
    "diff_huge_keys": lambda: lanedra(48, 64, [diff_attention(2, 1, 520, 24, 45, rot_dims=100)], [None]),
}


def lanedra_mixed():
    """Every branch together: order of layers, shared caches under other windows and constants, layers without feed-forward."""
    s = yarn(4.0, 96, 8.0, 0.7)
    return lanedra(88, 131, [
        diff_attention(6, 2, 20, 28, 24, base=5000.0, scaling=s),
        delta(4, 2, 24, 20, 4),
        diff_attention(6, 2, 20, 28, 57, base=5000.0, scaling=s, kv_from=0, diff=0.2, scale=0.35),
        delta(3, 3, 36, 44, 2),
        diff_attention(3, 3, 28, 12, 31, rot_dims=20, base=777.0, diff=0.7),
        diff_attention(6, 2, 20, 28, 11, base=5000.0, scaling=s, kv_from=0),
        delta(5, 1, 12, 60, 5)],
        [52, None, None, 68, 33, 40, 24], eps=2e-6, scale=2.5)


def window_needle(root, window, second=False, group=1, dim=24):
    """One attention layer in which token QUERY finds token KEY, through dimensions that are not rotated, with a score far above
    all others in one of the maps, wherever KEY stands inside the window."""
    kv, rot = 2, 8
    cfg = lanedra(64, 60, [diff_attention(kv * group, kv, dim, 40, window, rot_dims=rot, base=100.0, diff=0.3)], [None])
    w = lanedra_tensors(cfg, 78)
    w["l0.norm1b"] = w["l0.norm1b"] + 2.0
    m = cfg["layers"][0]["mixer"]
    h = plain.offset_norm(w["embed"] * cfg["embedding"]["scale"], w["l0.norm1"], cfg["norm"]["eps"])
    key = (w["l0.mix.k"] @ h[KEY]).reshape(kv, 2, dim)[..., rot:]
    q = w["l0.mix.q"].reshape(kv * group, 2, dim, -1)
    for head in range(kv * group):
        k = key[head // group, int(second)]
        q[head, int(second), rot:] += np.outer(k * (30.0 / m["scale"] / (k @ k)), h[QUERY] / (h[QUERY] @ h[QUERY]))
    return Model(root, cfg, weights=w)


def memory_model(root, conv=3, dim=20):
    """One delta layer without noticeable decay that writes at token KEY and next to nothing elsewhere: what stands in its state
    shows at every later token."""
    cfg = lanedra(64, 60, [delta(4, 2, dim, 24, conv)], [None])
    w = lanedra_tensors(cfg, 79)
    u = np.full(64, 64 ** -0.5)
    w["embed"] = w["embed"] - np.outer(w["embed"] @ u, u) + 10.0 * u
    w["embed"][KEY] -= 20.0 * u
    w["l0.norm1"] = np.zeros(64)
    w["l0.mix.b"] = np.tile(-1.3 * u, (4, 1))
    w["l0.mix.A_log"], w["l0.mix.dt_bias"] = np.full(4, -6.0), np.full(4, -4.0)
    w["l0.mix.a"] = w["l0.mix.a"] * 0.1
    return Model(root, cfg, weights=w)
