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


def offset_norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms_unit(x, eps) * (1.0 + np.asarray(w, F))


def yarn_frequencies(dims, base, scaling):
    """(frequency of every rotated pair, factor on cos and sin).  Pairs that turn more than ``fast`` times within the original
    context keep their frequency, those that turn less than ``slow`` times are divided by ``factor``, with a ramp between."""
    i = np.arange(dims // 2)
    f = np.asarray(base, F) ** (-2.0 * i / dims)
    if scaling is None:
        return f, 1.0

    def pair_of(turns):
        return dims * np.log(scaling["original"] / (2 * np.pi * turns)) / (2 * np.log(base))

    lo = max(np.floor(pair_of(scaling["fast"])), 0)
    hi = min(np.ceil(pair_of(scaling["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0, 1)
    return f / scaling["factor"] * ramp + f * (1 - ramp), 0.1 * np.log(scaling["factor"]) + 1.0


def rotate_half(x, positions, dims, freq, gain):
    """x [T, ..., D]: the pairs (i, i + dims/2) below ``dims`` turn by position * freq_i, scaled by gain; the rest passes."""
    out = np.array(x, F)
    h = dims // 2
    for t, p in enumerate(positions):
        c, s = np.cos(p * freq) * gain, np.sin(p * freq) * gain
        u, v = np.array(x[t, ..., :h]), np.array(x[t, ..., h:dims])
        out[t, ..., :h] = u * c - v * s
        out[t, ..., h:dims] = v * c + u * s
    return out


def unit_vectors(x):
    return x / np.sqrt(np.sum(np.square(x), axis=-1, keepdims=True) + 1e-6)


def delta_rule(q, k, v, decay, beta):
    """S <- decay_t S; u = beta_t (v_t - S^T k_t); S <- S + k_t u^T; o_t = S^T q_t.  q, k [T, H, N]; v [T, H, V]."""
    T, H, N = q.shape
    S = np.zeros((H, N, v.shape[2]))
    o = np.zeros(v.shape)
    for t in range(T):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hnv,hn->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hnv,hn->hv", S, q[t])
    return o


def delta(w, p, m, eps, x):
    H, G, D, V, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], x.shape[0]

    def mixed(name):
        taps = np.asarray(w[p + name + ".conv"], F)
        return silu(causal_conv(linear(w[p + name], x), taps, np.zeros(len(taps))))

    of = [h // (H // G) for h in range(H)]
    q = unit_vectors(mixed("q").reshape(T, G, D))[:, of] * D ** -0.5
    k = unit_vectors(mixed("k").reshape(T, G, D))[:, of]
    v = mixed("v").reshape(T, H, V)
    beta = sigmoid(linear(w[p + "b"], x))
    decay = np.exp(-np.exp(np.asarray(w[p + "A_log"], F)) * softplus(linear(w[p + "a"], x) + np.asarray(w[p + "dt_bias"], F)))
    o = rms_norm(delta_rule(q, k, v, decay, beta), w[p + "norm"], eps)
    return linear(w[p + "o"], o.reshape(T, H * V) * silu(linear(w[p + "g"], x)))


def rotated_maps(y, heads, m):
    """Projection rows [T, heads * 2 * dim] -> rotated [T, heads, 2 maps, dim]"""
    r = m["rot"]
    freq, gain = yarn_frequencies(r["dims"], r["base"], r.get("scaling"))
    return rotate_half(y.reshape(len(y), heads, 2, m["dim"]), np.arange(len(y)), r["dims"], freq, gain)


def attention_entries(w, p, m, x):
    """What an attention layer caches: (rotated keys [T, kv_heads, 2, dim], values [T, kv_heads, vdim])."""
    return rotated_maps(linear(w[p + "k"], x), m["kv_heads"], m), linear(w[p + "v"], x).reshape(len(x), m["kv_heads"], m["vdim"])


def visible(T, size):
    """[T, T]: position i sees j with 0 <= i - j < size"""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def softmax(scores):
    e = np.exp(scores - np.max(scores, axis=-1, keepdims=True))
    return e / np.sum(e, axis=-1, keepdims=True)


def map_lambda(w, p, diff):
    lq1, lk1, lq2, lk2 = (np.asarray(w[p + n], F) for n in ("lq1", "lk1", "lq2", "lk2"))
    return np.exp(lq1 @ lk1) - np.exp(lq2 @ lk2) + diff


def differential_attention(w, p, m, eps, x, entries):
    H, G, V, T = m["heads"], m["kv_heads"], m["vdim"], x.shape[0]
    k, v = entries
    q = rotated_maps(linear(w[p + "q"], x), H, m)
    seen = visible(T, m["mask"]["size"])
    out = np.zeros((T, H, V))
    for h in range(H):
        g = h // (H // G)
        a1, a2 = (softmax(np.where(seen, (q[:, h, i] @ k[:, g, i].T) * m["scale"], -np.inf)) @ v[:, g] for i in range(2))
        out[:, h] = a1 - map_lambda(w, p, m["diff"]) * a2
    return linear(w[p + "o"], (rms_unit(out, eps) * (1.0 - m["diff"])).reshape(T, H * V))


def forward_lanedra(config, w, tokens):
    eps = config["norm"]["eps"]
    x = np.asarray(w["embed"], F)[np.asarray(tokens)] * config["embedding"]["scale"]
    streams, cached = [], {}
    for i, L in enumerate(config["layers"]):
        p, m = f"l{i}.", L["mixer"]
        mp = p + "mix."
        h = offset_norm(x, w[p + "norm1"], eps)
        if L["type"] == "delta":
            y = delta(w, mp, m, eps, h)
        elif L["type"] == "attention":
            if "kv_from" not in m:
                cached[i] = attention_entries(w, mp, m, h)
            y = differential_attention(w, mp, m, eps, h, cached[m.get("kv_from", i)])
        else:
            raise ValueError(L["type"])
        x = x + offset_norm(y, w[p + "norm1b"], eps)
        if L.get("mlp") is not None:
            x = x + offset_norm(feed_forward(w, p + "mlp.", offset_norm(x, w[p + "norm2"], eps)), w[p + "norm2b"], eps)
        streams.append(x)
    return linear(w["head"], offset_norm(x, w["final.norm"], eps)), np.stack(streams)


def forward_vifivik(config, w, tokens):
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


FORWARD = {"Vifivik": forward_vifivik, "Lanedra": forward_lanedra}


def forward(config, w, tokens):
    """(logits [T, vocab], residual streams [layers, T, width])"""
    return FORWARD[config["architecture"]](config, w, tokens)
