"""Plain, slow float64 restatement (numpy) of the layer mechanisms of the config.json models: one function per mechanism,
written from the equations, no code shared with the product path.  Used by the tests only.

A whole sequence is evaluated at once; ``forward`` returns the logits and the residual stream after every layer.
``w`` maps tensor names to float arrays."""
from __future__ import annotations

import numpy as np

F = np.float64


def linear(W, x):
    return np.asarray(x, F) @ np.asarray(W, F).T


def sigmoid(z):
    z = np.asarray(z, F)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0, e) / (1.0 + e)


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def rms_unit(x, eps):
    return x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * np.asarray(w, F)


def rotate_interleaved(x, positions, dims, base):
    """x [T, ..., D]: the pairs (2i, 2i+1) below ``dims`` turn by position * base^(-2i/dims); the rest passes."""
    out = np.array(x, F)
    for t, p in enumerate(positions):
        for i in range(dims // 2):
            a = p * base ** (-2.0 * i / dims)
            u, v = np.array(x[t, ..., 2 * i]), np.array(x[t, ..., 2 * i + 1])
            out[t, ..., 2 * i] = u * np.cos(a) - v * np.sin(a)
            out[t, ..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, n] with the current token at the last tap; zeros before the first token."""
    T, C = x.shape
    n = taps.shape[1]
    pad = np.concatenate([np.zeros((n - 1, C)), x])
    y = np.zeros((T, C)) + np.asarray(bias, F)
    for t in range(T):
        for j in range(n):
            y[t] += taps[:, j] * pad[t + j]
    return y


def linear_recurrence(q, k, v, decay, weight):
    """S_t = decay_t S_(t-1) + weight_t k_t v_t^T, o_t = S_t^T q_t.  q, k [T, H, N]; v [T, H, V]; decay, weight [T, H]."""
    T, H, N = q.shape
    S = np.zeros((H, N, v.shape[2]))
    o = np.zeros(v.shape)
    for t in range(T):
        S = decay[t][:, None, None] * S + weight[t][:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hnv,hn->hv", S, q[t])
    return o


def mamba2(w, p, m, eps, x):
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, T = H * V, x.shape[0]
    u = linear(w[p + "in"], x)
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, np.asarray(w[p + "conv"], F), w[p + "conv.b"]))
    xs = xbc[:, :inner].reshape(T, H, V)
    group = [h // (H // G) for h in range(H)]
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)[:, group]
    C = xbc[:, inner + G * N:].reshape(T, G, N)[:, group]
    dt = softplus(dt + np.asarray(w[p + "dt_bias"], F))
    decay = np.exp(-np.exp(np.asarray(w[p + "A_log"], F)) * dt)
    y = linear_recurrence(C, B, xs, decay, dt) + np.asarray(w[p + "D"], F)[None, :, None] * xs
    y = y.reshape(T, inner) * silu(z)
    parts = m["norm_groups"]
    y = rms_unit(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * np.asarray(w[p + "norm"], F)
    return linear(w[p + "o"], y)


def retention(w, p, m, eps, x):
    H, D, V, T = m["heads"], m["dim"], m["vdim"], x.shape[0]
    q = linear(w[p + "q"], x).reshape(T, H, D)
    k = linear(w[p + "k"], x).reshape(T, H, D) * D ** -0.5
    v = linear(w[p + "v"], x).reshape(T, H, V)
    decay = np.tile(np.asarray(m["decay"], F), (T, 1))
    o = rms_unit(linear_recurrence(q, k, v, decay, np.ones((T, H))), eps).reshape(T, H * V)
    return linear(w[p + "o"], o * silu(linear(w[p + "g"], x)))


def latent_entries(w, p, m, eps, x):
    """What a latent-attention layer caches: (c [T, kv_rank], rotated shared key part [T, rot_dim])."""
    u = linear(w[p + "dkv"], x)
    R = m["kv_rank"]
    c = rms_norm(u[:, :R], w[p + "dkv.norm"], eps)
    return c, rotate_interleaved(u[:, R:], np.arange(len(x)), m["rot"]["dims"], m["rot"]["base"])


def sink_softmax(scores, sink):
    """scores [..., n] with -inf where masked; one more column exp(sink) in the denominator only."""
    top = np.maximum(np.max(scores, axis=-1, keepdims=True), sink)
    e = np.exp(scores - top)
    return e / (np.sum(e, axis=-1, keepdims=True) + np.exp(sink - top))


def latent_attention(w, p, m, eps, x, entries):
    H, D, R, V, T = m["heads"], m["dim"], m["rot_dim"], m["vdim"], x.shape[0]
    c, kr = entries
    q = linear(w[p + "q"], x).reshape(T, H, D + R)
    qr = rotate_interleaved(q[..., D:], np.arange(T), m["rot"]["dims"], m["rot"]["base"])
    k = linear(w[p + "uk"], c).reshape(T, H, D)
    v = linear(w[p + "uv"], c).reshape(T, H, V)
    gate = sigmoid(linear(w[p + "g"], x))
    out = np.zeros((T, H, V))
    seen = np.tril(np.ones((T, T), bool))
    for h in range(H):
        s = (q[:, h, :D] @ k[:, h].T + qr[:, h] @ kr.T) * m["scale"]
        out[:, h] = sink_softmax(np.where(seen, s, -np.inf), float(w[p + "sink"][h])) @ v[:, h]
    return linear(w[p + "o"], (out * gate[:, :, None]).reshape(T, H * V))


def feed_forward(w, p, x):
    return linear(w[p + "down"], silu(linear(w[p + "gate"], x)) * linear(w[p + "up"], x))


def forward(config, w, tokens):
    """(logits [T, vocab], residual streams [layers, T, width])"""
    eps = config["norm"]["eps"]
    x = np.asarray(w["embed"], F)[np.asarray(tokens)]
    streams, cached = [], {}
    for i, L in enumerate(config["layers"]):
        p, m = f"l{i}.", L["mixer"]
        mp = p + "mix."
        if L["type"] == "mamba2":
            y = mamba2(w, mp, m, eps, x)
        elif L["type"] == "retention":
            y = retention(w, mp, m, eps, x)
        elif L["type"] == "latent_attention":
            if "kv_from" not in m:
                cached[i] = latent_entries(w, mp, m, eps, x)
            y = latent_attention(w, mp, m, eps, x, cached[m.get("kv_from", i)])
        else:
            raise ValueError(L["type"])
        x = x + rms_norm(y, w[p + "norm1"], eps)
        if L.get("mlp") is not None:
            x = x + rms_norm(feed_forward(w, p + "mlp.", x), w[p + "norm2"], eps)
        streams.append(x)
    logits = linear(w["head"], rms_norm(x, w["final.norm"], eps))
    cap = config["logit_softcap"]
    return cap * np.tanh(logits / cap), np.stack(streams)
