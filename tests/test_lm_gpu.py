"""config.json models on the GPU against the plain float64 evaluation (oracle.lm_layers): every mechanism alone and all
together, prompts at any cut, token-by-token decoding, batches, slots that are used again, far keys, greedy generation
through the decode driver, the daemon and the trace runner -- in bfloat16 and in 32-bit."""
import json
import os
import subprocess

import numpy as np
import pytest

from tests import lm_models as lm

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
KIND = {True: "f32", False: "bf16"}
both = pytest.mark.parametrize("f32", [True, False], ids=KIND.get)


def driver(m, f32, batch=2, max_seq=400, **kw):
    from blackwell_b200.decode_driver import ModelDriver

    return ModelDriver(m.dir, batch=batch, max_seq=max_seq, f32=f32, use_graph=kw.pop("use_graph", False), **kw)


def run(d, slot, tokens, cuts):
    """Feeds the tokens in portions of the given sizes (the last one repeats)."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(cuts[min(i, len(cuts) - 1)], len(tokens) - at)
        out.append(d.portion(slot, tokens[at:at + n]))
        at, i = at + n, i + 1
    return np.concatenate(out)


def tokens_for(m, n, seed=0):
    return np.random.default_rng(seed).integers(0, m.cfg["vocab"], n)


# ----------------------------------------------------------------------------------------------- the matrix product
def _linear(x, W, T, N, K, x_f32, epilogue=0, cap=0.0, y_f32=1):
    import torch
    from blackwell_b200 import _lib
    import ctypes as C

    L = _lib.load()
    k8 = (K + 7) // 8 * 8
    wt = torch.zeros((N, k8), dtype=torch.bfloat16, device="cuda")
    wt[:, :K] = torch.from_numpy(W).to(torch.bfloat16)
    xt = torch.full((T, k8), 7.0, dtype=torch.float32 if x_f32 else torch.bfloat16, device="cuda")   # padding must not count
    xt[:, :K] = torch.from_numpy(x)
    cols = N // 2 if epilogue == 1 else N
    f32_out = x_f32 or (y_f32 and epilogue != 1)
    y = torch.full((T, cols + 3), -1.0, dtype=torch.float32 if f32_out else torch.bfloat16, device="cuda")
    e = L.bw_linear_bf16(C.c_void_p(y.data_ptr()), C.c_long(cols + 3), C.c_void_p(xt.data_ptr()), C.c_long(k8),
                         C.c_void_p(wt.data_ptr()), C.c_long(k8), T, N, K, int(y_f32), int(x_f32), epilogue, C.c_float(cap), None)
    assert e == 0
    torch.cuda.synchronize()
    y = y.float().cpu().numpy()
    assert (y[:, cols:] == -1.0).all()
    return y[:, :cols]


@pytest.mark.parametrize("T, stream_rows", [(t, 0) for t in (1, 2, 8, 9, 16, 20, 32, 33, 64, 65, 129, 300)] + [(t, 8) for t in (1, 2, 7, 8)])
@pytest.mark.parametrize("N, K", [(130, 40), (77, 200), (515, 328), (16, 1032)])
def test_linear_shapes(cuda, T, N, K, stream_rows):
    from blackwell_b200 import kernels

    kernels.set_tuning(23, stream_rows + 1)
    try:
        check_linear_shapes(T, N, K)
    finally:
        kernels.set_tuning(23, 0)


def check_linear_shapes(T, N, K):
    rng = np.random.default_rng(T * 1000 + N)
    _, W = lm.to_bf16(rng.standard_normal((N, K)))
    _, x = lm.to_bf16(rng.standard_normal((T, K)))
    want = x @ W.T
    got = _linear(x.astype(np.float32), W.astype(np.float32), T, N, K, False)
    assert np.abs(got - want).max() / np.abs(want).max() < 1e-5
    if T in (1, 20, 33, 300) and N % 2 == 0:
        g, u = want[:, 0::2], want[:, 1::2]
        sw = g / (1 + np.exp(-g)) * u
        got = _linear(x.astype(np.float32), W.astype(np.float32), T, N, K, False, epilogue=1)
        assert np.abs(got - sw).max() / np.abs(sw).max() < 5e-3
        got = _linear(x.astype(np.float32), W.astype(np.float32), T, N, K, True, epilogue=1)
        assert np.abs(got - sw).max() / np.abs(sw).max() < 1e-5
    if T in (8, 64, 129):
        cap = _linear(x.astype(np.float32), W.astype(np.float32), T, N, K, False, epilogue=2, cap=5.0)
        assert np.abs(cap - 5.0 * np.tanh(want / 5.0)).max() < 1e-4


@pytest.mark.parametrize("T, N, K", [(700, 2048, 512), (3000, 1400, 320), (4096, 4096, 192), (600, 26000, 1032), (40, 3000, 1024), (100, 20000, 264)])
def test_linear_large(cuda, T, N, K):
    rng = np.random.default_rng(T)
    _, W = lm.to_bf16(rng.standard_normal((N, K)).astype(np.float32))
    _, x = lm.to_bf16(rng.standard_normal((T, K)).astype(np.float32))
    want = x.astype(np.float32) @ W.astype(np.float32).T
    got = _linear(x.astype(np.float32), W.astype(np.float32), T, N, K, False)
    assert np.abs(got - want).max() / np.abs(want).max() < 1e-4


# ----------------------------------------------------------------------------------------------- mechanisms, cuts
@both
@pytest.mark.parametrize("name", lm.SINGLE)
def test_mechanism_alone(cuda, tmp_path, name, f32):
    m = lm.Model(tmp_path, lm.SINGLE[name](), 5)
    tok = tokens_for(m, 150)
    want, bar = m.plain(tok)[0], m.bar(tok, f32)
    d = driver(m, f32)
    for slot, cuts in ((0, [150]), (1, [1]), (0, [2, 3, 70, 17, 1, 40])):
        d.release(slot)
        err = lm.rel_error(run(d, slot, tok, cuts), want)
        assert err.max() < bar, (cuts[:3], int(err.argmax()), err.max(), bar)
    d.close()


@pytest.mark.parametrize("vdim", [40, 100])
def test_long_prompt_many_heads(cuda, tmp_path, vdim):
    """Prompts long enough for the attention kernel's tall blocks, cut in unequal parts and whole."""
    m = lm.Model(tmp_path, lm.config(40, 50, [lm.latent(40, 12, 6, 24, vdim, 0.3)], [None]), 4)
    tok = tokens_for(m, 1100)
    want, bar = m.plain(tok)[0], m.bar(tok, False)
    d = driver(m, False, max_seq=1100)
    for cuts in ([1100], [37, 1063], [1030, 17, 1]):
        d.release(0)
        err = lm.rel_error(run(d, 0, tok, cuts), want)
        assert err.max() < bar, (cuts, int(err.argmax()), err.max(), bar)
    d.close()


@both
def test_layers_one_by_one(cuda, tmp_path, f32):
    m = lm.Model(tmp_path, lm.mixed(), 6)
    tok = tokens_for(m, 40)
    streams = m.plain(tok)[1]
    d = driver(m, f32)
    buf = d.watch(40)
    for cuts in ([40], [1], [33, 2, 5]):
        d.release(0)
        at, got = 0, []
        for n in cuts * 40:
            n = min(n, 40 - at)
            if n == 0:
                break
            d.portion(0, tok[at:at + n], want=[])
            got.append(buf[:, :n].cpu().numpy())
            at += n
        err = np.abs(np.concatenate(got, 1) - streams).max((1, 2)) / np.abs(streams).max((1, 2))
        assert err.max() < (3e-6 if f32 else 0.05), err
    d.watch(0)
    d.close()


@both
@pytest.mark.parametrize("cuts", [[260], [1], [2], [2, 62, 64, 65, 1, 3], [17, 100, 16], [64], [63, 1, 129]], ids=str)
def test_portions(cuda, tmp_path, cuts, f32):
    m = lm.Model(tmp_path, lm.mixed(), 7)
    tok = tokens_for(m, 260, 3)
    d = driver(m, f32)
    err = lm.rel_error(run(d, 1, tok, cuts), m.plain(tok)[0])
    bar = m.bar(tok, f32)
    assert err.max() < bar, (int(err.argmax()), err.max(), bar)
    assert d.held(1) == 260 and d.held(0) == 0
    d.close()


@both
def test_long_portion_is_split_inside(cuda, tmp_path, f32):
    m = lm.Model(tmp_path, lm.mixed(), 7)
    tok = tokens_for(m, 101, 4)
    want, bar = m.plain(tok)[0], m.bar(tok, f32)
    for rows in (1, 5, 40):
        d = driver(m, f32, max_portion=rows)
        assert lm.rel_error(d.portion(0, tok), want).max() < bar
        d.close()


@both
def test_wanted_places(cuda, tmp_path, f32):
    m = lm.Model(tmp_path, lm.mixed(), 8)
    tok = tokens_for(m, 200, 5)
    d = driver(m, f32)
    every = d.portion(0, tok)
    some = d.portion(1, tok, want=[0, 63, 64, 199])
    assert some.shape == (4, m.cfg["vocab"]) and lm.rel_error(some, every[[0, 63, 64, 199]]).max() < 1e-6
    d.close()


@both
def test_softcap_may_be_absent(cuda, tmp_path, f32):
    cfg = lm.mixed()
    cfg["logit_softcap"] = 1e6      # the plain evaluation's limit of no cap
    m = lm.Model(tmp_path, cfg, 9)
    cfg = json.loads(json.dumps(cfg))
    cfg["logit_softcap"] = None
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    tok = tokens_for(m, 20)
    d = driver(m, f32)
    assert lm.rel_error(d.portion(0, tok), m.plain(tok)[0]).max() < m.bar(tok, f32)
    d.close()


# ----------------------------------------------------------------------------------------------- far keys
@both
@pytest.mark.parametrize("rank, heads", [(40, 3), (200, 18)])
def test_needle(cuda, tmp_path, rank, heads, f32):
    m = lm.needle_model(tmp_path, rank, heads)
    d = driver(m, f32, max_seq=700)
    for key_at in (0, 1, 15, 63, 64, 127, 128, 319):
        # QUERY just before KEY (must not see it), just after, and far away; the far ones both in a prompt and decoded
        tok = lm.needle_tokens(330, key_at, [p for p in (key_at - 1, key_at + 1, 325, 329) if p >= 0], seed=key_at)
        want, bar = m.plain(tok)[0], m.bar(tok, f32)
        assert bar < (1e-4 if f32 else 0.15)
        for cuts in ([330], [key_at + 1, 329], [326, 1], [key_at or 1, 2, 64]):
            d.release(0)
            err = lm.rel_error(run(d, 0, tok, cuts), want)
            assert err.max() < bar, (key_at, cuts, int(err.argmax()), err.max(), bar)
    d.close()


@both
def test_strong_sink(cuda, tmp_path, f32):
    m = lm.needle_model(tmp_path)
    w = {k: np.array(v) for k, v in m.w.items()}
    w["l0.mix.sink"] = np.array([45.0, -45.0, 38.0])    # above, below and about the needle's score
    m = lm.Model(tmp_path / "sink", m.cfg, weights=w)
    tok = lm.needle_tokens(200, 70, [90, 199])
    want, bar = m.plain(tok)[0], m.bar(tok, f32)
    d = driver(m, f32)
    for slot, cuts in ((0, [200]), (1, [1]), (0, [150, 2, 1])):
        d.release(slot)
        assert lm.rel_error(run(d, slot, tok, cuts), want).max() < bar
    d.close()


# ----------------------------------------------------------------------------------------------- slots, batches, decoding
@both
def test_slots_are_used_again(cuda, tmp_path, f32):
    m = lm.Model(tmp_path, lm.mixed(), 10)
    first, second = tokens_for(m, 180, 1), tokens_for(m, 60, 2)
    d = driver(m, f32, batch=3)
    for slot in range(3):
        run(d, slot, first, [100, 1, 7])
    fresh = driver(m, f32, batch=1)
    want = run(fresh, 0, second, [30, 2, 1])
    for slot in (2, 0):
        d.release(slot)
        assert np.array_equal(run(d, slot, second, [30, 2, 1]), want)
    # the slot in between still holds its sequence
    tail = tokens_for(m, 20, 3)
    got = run(d, 1, tail, [1])
    both_parts = np.concatenate([first, tail])
    assert lm.rel_error(got, m.plain(both_parts)[0][180:]).max() < m.bar(both_parts, f32)
    fresh.close()
    d.close()


@both
def test_interleaved_sequences(cuda, tmp_path, f32):
    m = lm.Model(tmp_path, lm.mixed(), 12)
    seqs = [tokens_for(m, n, 20 + n) for n in (90, 33, 140)]
    d = driver(m, f32, batch=3)
    got, at = [[], [], []], [0, 0, 0]
    rng = np.random.default_rng(0)
    while any(at[i] < len(s) for i, s in enumerate(seqs)):
        i = int(rng.integers(3))
        n = min(int(rng.choice([1, 2, 5, 30])), len(seqs[i]) - at[i])
        if n:
            got[i].append(d.portion(i, seqs[i][at[i]:at[i] + n]))
            at[i] += n
    for i, s in enumerate(seqs):
        assert lm.rel_error(np.concatenate(got[i]), m.plain(s)[0]).max() < m.bar(s, f32)
    d.close()


@both
def test_long_decoding(cuda, tmp_path, f32):
    m = lm.Model(tmp_path, lm.mixed(), 13)
    tok = tokens_for(m, 330, 6)
    d = driver(m, f32)
    err = lm.rel_error(run(d, 0, tok, [30] + [1] * 300), m.plain(tok)[0])
    assert err.max() < m.bar(tok, f32) and err[300:].mean() < 3 * err[:60].mean() + 1e-6
    d.close()


@pytest.mark.parametrize("graph", [True, False])
@pytest.mark.parametrize("batch", [1, 3, 11, 20])
def test_greedy_generation_matches_plain(cuda, tmp_path, batch, graph):
    """32-bit greedy generation of unequal prompts through begin / step / result: the ids of the plain evaluation."""
    m = lm.Model(tmp_path, lm.mixed(), 14)
    lens = [1, 37, 2, 90, 5, 64, 65, 3, 16, 17, 33, 8, 1, 120, 50, 4, 6, 7, 9, 10][:batch]
    prompts = [tokens_for(m, n, 100 + i).tolist() for i, n in enumerate(lens)]
    d = driver(m, True, batch=batch, max_seq=160, max_prompt=130, max_new=8, use_graph=graph)
    for _ in range(2):   # the second generation uses the slots again
        d.begin(prompts)
        for _ in range(d.steps(max(lens), 6)):
            d.step()
        got = d.result()[:, :6]
    for i in list(range(batch))[:6]:
        assert got[i].tolist() == m.greedy(prompts[i], 6), i
    d.close()


@both
def test_batch_against_each_alone(cuda, tmp_path, f32):
    """The step's logits of a sequence do not depend on its neighbours, and equal the plain ones."""
    import torch

    m = lm.Model(tmp_path, lm.mixed(), 15)
    lens = [70, 3, 1, 130, 40, 9, 64, 2, 20, 31]
    prompts = [tokens_for(m, n, 200 + i).tolist() for i, n in enumerate(lens)]
    d = driver(m, f32, batch=len(lens), max_seq=200, max_prompt=130, max_new=8, use_graph=True)
    d.begin(prompts)
    steps = []
    for _ in range(5):
        d.step()
        torch.cuda.synchronize()
        steps.append(d.logits().cpu().numpy().copy())
    ids = d.result()
    for i, p in enumerate(prompts):
        seq = p + ids[i, :4].tolist()
        want, bar = m.plain(seq)[0][len(p) - 1:], m.bar(seq, f32)
        got = np.stack([s[i] for s in steps])
        assert lm.rel_error(got, want).max() < bar, i
        alone = driver(m, f32, batch=1, max_seq=200)
        single = np.concatenate([alone.portion(0, [t]) for t in seq])[len(p) - 1:] if len(p) < 10 else alone.portion(0, seq)[len(p) - 1:]
        assert lm.rel_error(got, single).max() < bar, i
        alone.close()
    d.close()


def test_rejected_calls(cuda, tmp_path):
    from blackwell_b200.kernels import KernelError

    m = lm.Model(tmp_path, lm.mixed(), 16)
    d = driver(m, False, max_seq=30)
    for slot, tok in ((2, [1]), (-1, [1]), (0, [131]), (0, [-1]), (0, [1] * 31)):
        with pytest.raises(KernelError):
            d.portion(slot, tok)
    with pytest.raises(KernelError):
        d.portion(0, [1, 2, 3], want=[2, 1])
    d.portion(0, [1] * 29, want=[])
    with pytest.raises(KernelError):
        d.portion(0, [1, 1])
    d.close()
    (tmp_path / "config.json").write_text(json.dumps({**m.cfg, "width": 96}))    # sizes that the weights do not have
    with pytest.raises(KernelError):
        driver(m, False)


# ----------------------------------------------------------------------------------------------- programs
def test_daemon_generates_from_ids(cuda, tmp_path):
    m = lm.Model(tmp_path / "m", lm.mixed(), 17)
    prompts = [tokens_for(m, n, 300 + n).tolist() for n in (5, 40, 1)]
    exe = os.path.join(ROOT, "blackwell_b200", "lib", "inference_server_w4a8")
    reqs = [{"prompt_ids": prompts, "max_tokens": 4}, {"prompt_ids": [prompts[0]], "max_tokens": 2}, {"prompt_ids": [[999]], "max_tokens": 2}]
    p = subprocess.run([exe, "--weights", m.dir, "--batch", "2", "--max-seq", "128", "--dtype", "float32"],
                       input="".join(json.dumps(r) + "\n" for r in reqs), capture_output=True, text=True, timeout=120)
    out = [json.loads(x) for x in p.stdout.splitlines()]
    assert p.returncode == 0 and len(out) == 3, p.stderr[-2000:]
    for got, prompt in zip(out[0]["tokens"], prompts):
        assert got == m.greedy(prompt, 5)
    assert out[1]["tokens"][0] == out[0]["tokens"][0][:3] and "error" in out[2]


@both
def test_trace_runner(cuda, tmp_path, f32):
    m = lm.Model(tmp_path / "m", lm.mixed(), 18)
    out = tmp_path / "out"
    out.mkdir()
    a, b = tokens_for(m, 80, 1).tolist(), tokens_for(m, 25, 2).tolist()
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 49]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b[:2], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "a", "tokens": a[50:51], "want": [0]}, {"id": "b", "tokens": b[2:], "want": [3, 22]}], "end": ["b"]},
        {"step": 3, "entries": [{"id": "a", "tokens": a[51:], "want": [28]}], "end": ["a"]},
        {"step": 4, "entries": [{"id": "a", "tokens": b, "want": [24]}], "end": ["a"]},
    ]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", m.dir, "--dtype", "float32" if f32 else "bfloat16",
                        "--out", str(out), "--max-tokens", "128"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    wa, wb = m.plain(a)[0], m.plain(b)[0]
    rows = {0: wa[[0, 49]], 2: np.concatenate([wa[[50]], wb[[5, 24]]]), 3: wa[[79]], 4: wb[[24]]}
    assert not (out / "1.f32").exists()
    for i, want in rows.items():
        got = np.fromfile(out / f"{i}.f32", "<f4").reshape(want.shape)
        assert lm.rel_error(got, want).max() < m.bar(a, f32)
