"""Lanedra configurations without a GPU: the reader, and the plain evaluation that the GPU tests compare with -- including
that it sees the faults those tests are there to find (each fault is planted in the plain evaluation)."""
import copy
import json

import numpy as np
import pytest

from oracle import lm_layers as plain
from tests import lm_models as lm
from tests.test_lm_cpu import probe


def test_probe_counts_layers(tmp_path):
    info = probe(tmp_path, lm.lanedra_mixed())
    assert (info.architecture, info.layers, info.width, info.vocab) == (b"Lanedra", 7, 88, 131)
    assert (info.delta_layers, info.diff_attention_layers, info.shared_cache_layers) == (3, 4, 2)
    assert (info.mamba2_layers, info.retention_layers, info.latent_layers) == (0, 0, 0)


@pytest.mark.parametrize("name", lm.LANEDRA)
def test_probe_accepts(tmp_path, name):
    assert probe(tmp_path, lm.LANEDRA[name]()).layers == 1


@pytest.mark.parametrize("change, message", [
    (lambda c: c.pop("embedding"), "'embedding'"),
    (lambda c: c["layers"][1].update(type="mamba2"), "unknown type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "'kv_heads'"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "'conv'"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "'diff'"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "'size'"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=22), "'dims'"),
    (lambda c: c["layers"][4]["mixer"]["rot"].update(dims=7), "bad rotation"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "'slow'"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), "scaling"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][5]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=24), "kv_from"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(base=4999.0), "kv_from"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "feed-forward"),
])
def test_probe_rejects(tmp_path, change, message):
    cfg = lm.lanedra_mixed()
    change(cfg)
    with pytest.raises(ValueError, match=message):
        probe(tmp_path, cfg)


def test_plain_evaluation_is_causal(tmp_path):
    m = lm.Model(tmp_path, lm.lanedra_mixed(), 3)
    tok = np.random.default_rng(0).integers(0, 131, 24)
    whole = m.plain(tok)[0]
    for n in (1, 2, 9):
        assert np.abs(m.plain(tok[:n])[0] - whole[:n]).max() < 1e-9


def test_plain_delta_rule_overwrites():
    """With full strength and no decay the last value written under a key is what the key finds; orthogonal keys stay."""
    k = np.eye(3)[[0, 1, 0, 2]][:, None, :]
    v = np.arange(8.0).reshape(4, 1, 2)
    o = plain.delta_rule(np.eye(3)[[0, 0, 0, 1]][:, None, :], k, v, np.ones((4, 1)), np.ones((4, 1)))
    assert np.allclose(o[:, 0], v[[0, 0, 2, 1], 0])


def test_plain_delta_rule_triangular_form():
    """The writes of a run of tokens solve one unit lower triangular system (the form the prompt kernels use)."""
    rng = np.random.default_rng(1)
    T, N, V = 9, 4, 3
    q, k = (plain.unit_vectors(rng.standard_normal((T, 1, N))) for _ in range(2))
    v, g, b = rng.standard_normal((T, 1, V)), rng.uniform(0.4, 1, (T, 1)), rng.uniform(0, 1, (T, 1))
    o = plain.delta_rule(q, k, v, g, b)[:, 0]
    G = np.cumprod(g[:, 0])
    ratio = np.tril(G[:, None] / G[None, :])
    A = np.tril(b * ratio * (k[:, 0] @ k[:, 0].T), -1)
    u = np.linalg.solve(np.eye(T) + A, b * v[:, 0])
    assert np.allclose(o, (ratio * (q[:, 0] @ k[:, 0].T)) @ u)


def test_plain_yarn_frequencies():
    f, gain = plain.yarn_frequencies(16, 10000.0, None)
    assert gain == 1.0 and np.allclose(f, 10000.0 ** (-np.arange(8) / 8))
    s, gain = plain.yarn_frequencies(16, 10000.0, lm.yarn(8.0, 4096, 32.0, 1.0))
    assert np.isclose(gain, 1 + 0.1 * np.log(8.0)) and np.allclose(s[:2], f[:2]) and np.allclose(s[-1], f[-1] / 8.0)
    assert (np.diff(s / f) <= 1e-12).all() and ((s / f > 1 / 8 + 1e-6) & (s / f < 1 - 1e-6)).any()


def test_plain_rotation_depends_on_distance_only():
    rng = np.random.default_rng(2)
    q, k = rng.standard_normal((2, 1, 10))
    f, gain = plain.yarn_frequencies(6, 100.0, lm.yarn(4.0, 50, 4.0, 0.5))
    dots = [plain.rotate_half(q, [p + 7], 6, f, gain)[0] @ plain.rotate_half(k, [p], 6, f, gain)[0] for p in (0, 5, 90)]
    assert np.allclose(dots, dots[0])


def cut(f, n=20):
    return lambda *a: np.concatenate([f(*(x[:n] for x in a)), f(*(x[n:] for x in a))])


FAULTS = {
    "state lost between portions": ("delta_rule", cut),
    "convolution inputs lost between portions": ("causal_conv", lambda f: lambda x, t, b: np.concatenate([f(x[:20], t, b), f(x[20:], t, b)])),
    "read-out before the write": ("delta_rule", lambda f: lambda q, k, v, g, b: f(
        q, k, v, g, b) - b[..., None] * np.sum(q * k, -1, keepdims=True) * v),
    "decay after the write": ("delta_rule", lambda f: lambda q, k, v, g, b: f(q, k, v, np.concatenate([np.ones_like(g[:1]), g[:-1]]), b)),
    "nothing taken off the value": ("delta_rule", lambda f: lambda q, k, v, g, b: plain.linear_recurrence(q, k, v, g, b)),
    "keys not of unit length": ("unit_vectors", lambda f: lambda x: x),
    "positions start again": ("rotate_half", lambda f: lambda x, p, *a: f(x, np.asarray(p) % 20, *a)),
    "interleaved rotation": ("rotate_half", lambda f: lambda x, p, d, fr, g: np.concatenate(
        [plain.rotate_interleaved(x, p, d, 5000.0)[..., :d], x[..., d:]], -1)),
    "frequencies not scaled": ("yarn_frequencies", lambda f: lambda d, b, s: (f(d, b, None)[0], f(d, b, s)[1])),
    "cos and sin not scaled": ("yarn_frequencies", lambda f: lambda d, b, s: (f(d, b, s)[0], 1.0)),
    "window one longer": ("visible", lambda f: lambda T, n: f(T, n + 1)),
    "window one shorter": ("visible", lambda f: lambda T, n: f(T, n - 1)),
    "second map not weighted by lambda": ("map_lambda", lambda f: lambda w, p, d: f(w, p, d) + 0.3),
    "second map left out": ("map_lambda", lambda f: lambda w, p, d: 0.0),
    "norms without the offset": ("offset_norm", lambda f: lambda x, w, eps: plain.rms_norm(x, w, eps)),
}


@pytest.mark.parametrize("fault", FAULTS)
def test_faults_show_in_the_logits(tmp_path, monkeypatch, fault):
    m = lm.Model(tmp_path, lm.lanedra_mixed(), 11)
    tok = np.random.default_rng(2).integers(0, 131, 60)
    good = m.plain(tok)[0]
    name, make = FAULTS[fault]
    monkeypatch.setattr(plain, name, make(getattr(plain, name)))
    bad = m.plain(tok)[0]
    assert lm.rel_error(bad[20:], good[20:]).max() > 0.1   # thousands of times the bars of the 32-bit tests


@pytest.mark.parametrize("window, second", [(50, False), (16, True), (129, True)])
def test_window_needle_shows_one_position(tmp_path, monkeypatch, window, second):
    """The last position that sees the key and the first that does not differ, and an edge that is off by one shows there only."""
    m = lm.window_needle(tmp_path, window, second)
    at = [40 + window - 1, 40 + window]
    tok = lm.needle_tokens(200, 40, at)
    good = m.plain(tok)[0]
    visible = plain.visible
    for d, place in ((1, at[1]), (-1, at[0])):
        monkeypatch.setattr(plain, "visible", lambda T, n: visible(T, n + d))
        err = lm.rel_error(m.plain(tok)[0], good)
        assert err[place] > 0.3 and err[place] > 3 * m.bar(tok, False)
    monkeypatch.setattr(plain, "visible", visible)


def test_memory_model_remembers(tmp_path):
    m = lm.memory_model(tmp_path)
    tok = lm.needle_tokens(250, 5, [])
    other = tok.copy()
    other[5] = 9
    err = lm.rel_error(m.plain(other)[0], m.plain(tok)[0])
    assert err[:5].max() < 1e-9 and err[5:].min() > 2e-3 and np.median(err[150:]) > 0.1


def test_kv_from_reads_the_other_layers_cache(tmp_path):
    """The shared cache must be the owner's: with keys and values of its own the answer changes."""
    m = lm.Model(tmp_path, lm.lanedra_mixed(), 5)
    tok = np.random.default_rng(4).integers(0, 131, 12)
    good = m.plain(tok)[0]
    cfg = copy.deepcopy(m.cfg)
    cfg["layers"][5]["mixer"].pop("kv_from")
    w = dict(m.w)
    w["l5.mix.k"], w["l5.mix.v"] = w["l0.mix.k"], w["l0.mix.v"]
    assert lm.rel_error(plain.forward(cfg, w, tok)[0], good).max() > 0.02
    assert json.dumps(cfg) != json.dumps(m.cfg)
