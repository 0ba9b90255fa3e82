"""config.json models without a GPU: the reader of configurations, and the plain evaluation that the GPU tests compare
with -- including that it sees the faults those tests are there to find (each fault is planted in the plain
evaluation)."""
import copy
import json

import numpy as np
import pytest

from oracle import lm_layers as plain
from tests import lm_models as lm


def probe(tmp_path, cfg):
    from blackwell_b200.decode_driver import probe_model

    (tmp_path / "config.json").write_text(cfg if isinstance(cfg, str) else json.dumps(cfg))
    return probe_model(str(tmp_path))


def test_probe_counts_layers(tmp_path):
    info = probe(tmp_path, lm.mixed())
    assert (info.architecture, info.layers, info.width, info.vocab) == (b"Vifivik", 8, 88, 131)
    assert (info.mamba2_layers, info.retention_layers, info.latent_layers, info.shared_cache_layers) == (2, 2, 4, 2)


@pytest.mark.parametrize("change, message", [
    (lambda c: c.update(architecture="Other"), "not known"),
    (lambda c: c.pop("architecture"), "names no architecture"),
    (lambda c: c.pop("width"), "'width'"),
    (lambda c: c["layers"][1].update(type="mamba9"), "unknown type"),
    (lambda c: c["layers"][1]["mixer"].update(groups=3), "'groups'"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=7), "'norm_groups'"),
    (lambda c: c["layers"][3]["mixer"].update(decay=[0.5]), "'decay'"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][6]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=48), "kv_from"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=12), "'dims'"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "feed-forward"),
    (lambda c: c["layers"][0]["mixer"].update(heads=2.5), "'heads'"),
])
def test_probe_rejects(tmp_path, change, message):
    cfg = lm.mixed()
    change(cfg)
    with pytest.raises(ValueError, match=message):
        probe(tmp_path, cfg)


def test_probe_rejects_broken_files(tmp_path):
    with pytest.raises(ValueError, match="malformed"):
        probe(tmp_path, '{"architecture": "Vifivik", ')
    from blackwell_b200.decode_driver import probe_model

    with pytest.raises(ValueError, match="cannot open"):
        probe_model(str(tmp_path / "nowhere"))


def test_plain_evaluation_is_causal(tmp_path):
    m = lm.Model(tmp_path, lm.mixed(), 3)
    tok = np.random.default_rng(0).integers(0, 131, 24)
    whole = m.plain(tok)[0]
    for n in (1, 2, 9):
        assert np.abs(m.plain(tok[:n])[0] - whole[:n]).max() < 1e-9


def test_plain_recurrence_closed_form():
    rng = np.random.default_rng(1)
    T, H, N, V = 7, 2, 3, 4
    q, k, v = (rng.standard_normal((T, H, n)) for n in (N, N, V))
    a, w = rng.uniform(0.5, 1, (T, H)), rng.uniform(0.1, 2, (T, H))
    o = plain.linear_recurrence(q, k, v, a, w)
    for t in range(T):
        for h in range(H):
            want = sum(np.prod(a[s + 1:t + 1, h]) * w[s, h] * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1))
            assert np.allclose(o[t, h], want)


def test_plain_sink_takes_weight_but_gives_nothing():
    p = plain.sink_softmax(np.array([0.0, -np.inf, 1.0]), 1.0)
    e = np.exp(1.0)
    assert np.allclose(p, [1 / (1 + 2 * e), 0, e / (1 + 2 * e)])


FAULTS = {
    "state lost between portions": ("linear_recurrence", lambda f: lambda q, k, v, a, w: np.concatenate(
        [f(q[:20], k[:20], v[:20], a[:20], w[:20]), f(q[20:], k[20:], v[20:], a[20:], w[20:])])),
    "convolution inputs lost between portions": ("causal_conv", lambda f: lambda x, t, b: np.concatenate(
        [f(x[:20], t, b), f(x[20:], t, b)])),
    "positions start again": ("rotate_interleaved", lambda f: lambda x, p, d, b: f(x, np.asarray(p) % 20, d, b)),
    "half-split rotation": ("rotate_interleaved", lambda f: lambda x, p, d, b: np.concatenate(
        [f(np.stack([x[..., :d // 2], x[..., d // 2:d]], -1).reshape(x.shape[:-1] + (d,)), p, d, b)[..., 0::2],
         f(np.stack([x[..., :d // 2], x[..., d // 2:d]], -1).reshape(x.shape[:-1] + (d,)), p, d, b)[..., 1::2]], -1)),
    "no sink": ("sink_softmax", lambda f: lambda s, sink: f(s, -1e9)),
    "scaled sink": ("sink_softmax", lambda f: lambda s, sink: f(s, 0.3 * sink)),
    "newest key missing": ("sink_softmax", lambda f: lambda s, sink: f(
        np.where(np.eye(len(s), dtype=bool) & (np.arange(len(s)) > 0)[:, None], -np.inf, s), sink)),
    "unit norm without eps": ("rms_unit", lambda f: lambda x, eps: f(x, 0.3)),
}


@pytest.mark.parametrize("fault", FAULTS)
def test_faults_show_in_the_logits(tmp_path, monkeypatch, fault):
    m = lm.Model(tmp_path, lm.mixed(), 11)
    tok = np.random.default_rng(2).integers(0, 131, 40)
    good = m.plain(tok)[0]
    name, make = FAULTS[fault]
    monkeypatch.setattr(plain, name, make(getattr(plain, name)))
    bad = m.plain(tok)[0]
    assert lm.rel_error(bad[20:], good[20:]).max() > 0.1   # far beyond the bars of the GPU tests


def test_kv_from_reads_the_other_layers_cache(tmp_path):
    """The shared cache must be the owner's: with another latent the answer changes."""
    m = lm.Model(tmp_path, lm.mixed(), 5)
    tok = np.random.default_rng(4).integers(0, 131, 12)
    good = m.plain(tok)[0]
    cfg = copy.deepcopy(m.cfg)
    cfg["layers"][6]["mixer"].pop("kv_from")
    w = dict(m.w)
    w["l6.mix.dkv"], w["l6.mix.dkv.norm"] = w["l0.mix.dkv"], w["l0.mix.dkv.norm"]
    assert lm.rel_error(plain.forward(cfg, w, tok)[0], good).max() > 0.02


@pytest.mark.parametrize("key_at, query_at", [(0, 199), (63, 199), (64, 65), (128, 199)])
def test_needle_shows_one_missing_key(tmp_path, monkeypatch, key_at, query_at):
    m = lm.needle_model(tmp_path)
    tok = lm.needle_tokens(200, key_at, query_at)
    good = m.plain(tok)[0]
    softmax = plain.sink_softmax

    def without(s, sink):
        s = s.copy()
        s[query_at, key_at] = -np.inf
        return softmax(s, sink)

    monkeypatch.setattr(plain, "sink_softmax", without)
    err = lm.rel_error(m.plain(tok)[0], good)
    assert err[query_at] > 0.3 and np.delete(err, query_at).max() < 1e-9
