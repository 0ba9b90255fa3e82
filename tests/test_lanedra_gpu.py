"""Lanedra models on the GPU against the plain float64 evaluation (oracle.lm_layers): gated delta rule and windowed
differential attention alone and together, prompts at any cut, token-by-token decoding, batches, slots that are used again,
keys at the edges of every window, memory far back, greedy generation through the decode driver, the daemon and the trace
runner -- in bfloat16 and in 32-bit."""
import ctypes as C
import json
import os
import subprocess

import numpy as np
import pytest

from oracle import lm_layers as plain
from tests import lm_models as lm
from tests.test_lm_gpu import ROOT, both, driver, run, tokens_for

pytestmark = pytest.mark.gpu


def check(m, d, tok, cuts_list, f32, slots=(0, 1)):
    want, bar = m.plain(tok)[0], m.bar(tok, f32)
    for i, cuts in enumerate(cuts_list):
        slot = slots[i % len(slots)]
        d.release(slot)
        err = lm.rel_error(run(d, slot, tok, cuts), want)
        assert err.max() < bar, (cuts[:3], int(err.argmax()), err.max(), bar)


# ----------------------------------------------------------------------------------------------- mechanisms, cuts
@both
@pytest.mark.parametrize("name", lm.LANEDRA)
def test_mechanism_alone(cuda, tmp_path, name, f32):
    m = lm.Model(tmp_path, lm.LANEDRA[name](), 5)
    d = driver(m, f32)
    check(m, d, tokens_for(m, 150), ([150], [1], [2, 3, 70, 17, 1, 40]), f32)
    d.close()


@pytest.mark.parametrize("vdim, window", [(40, 300), (40, 2000), (100, 250), (200, 130)])
def test_long_prompt_many_heads(cuda, tmp_path, vdim, window):
    """Prompts long enough for the attention kernel's tall blocks, cut in unequal parts and whole."""
    m = lm.Model(tmp_path, lm.lanedra(40, 50, [lm.diff_attention(20, 5, 20, vdim, window)], [None]), 4)
    tok = tokens_for(m, 1100)
    d = driver(m, False, max_seq=1100)
    check(m, d, tok, ([1100], [37, 1063], [1030, 17, 1]), False)
    d.close()


def test_long_delta_prompt(cuda, tmp_path):
    m = lm.Model(tmp_path, lm.lanedra(40, 50, [lm.delta(6, 2, 40, 72, 4)], [None]), 4)
    tok = tokens_for(m, 1100)
    d = driver(m, False, max_seq=1100)
    check(m, d, tok, ([1100], [37, 1063], [1030, 17, 1]), False)
    d.close()


@both
def test_layers_one_by_one(cuda, tmp_path, f32):
    m = lm.Model(tmp_path, lm.lanedra_mixed(), 6)
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
        assert err.max() < (2e-5 if f32 else 0.1), err
    d.watch(0)
    d.close()


@both
@pytest.mark.parametrize("cuts", [[260], [1], [2], [2, 62, 64, 65, 1, 3], [17, 100, 16], [64], [63, 1, 129]], ids=str)
def test_portions(cuda, tmp_path, cuts, f32):
    m = lm.Model(tmp_path, lm.lanedra_mixed(), 7)
    tok = tokens_for(m, 260, 3)
    d = driver(m, f32)
    check(m, d, tok, [cuts], f32, slots=(1,))
    assert d.held(1) == 260 and d.held(0) == 0
    d.close()


@both
@pytest.mark.parametrize("rows", [1, 5, 20, 40])
def test_small_rings(cuda, tmp_path, rows, f32):
    """Caches that hold little more than the longest window: every row is overwritten many times, by portions of all sizes."""
    m = lm.Model(tmp_path, lm.lanedra_mixed(), 7)
    d = driver(m, f32, max_portion=rows)
    check(m, d, tokens_for(m, 230, 4), ([230], [1], [rows, 1, 3, 100, 2]), f32)
    d.close()


@both
def test_wanted_places(cuda, tmp_path, f32):
    m = lm.Model(tmp_path, lm.lanedra_mixed(), 8)
    tok = tokens_for(m, 200, 5)
    d = driver(m, f32)
    every = d.portion(0, tok)
    some = d.portion(1, tok, want=[0, 63, 64, 199])
    assert some.shape == (4, m.cfg["vocab"]) and lm.rel_error(some, every[[0, 63, 64, 199]]).max() < 1e-6
    d.close()


# ----------------------------------------------------------------------------------------------- windows, memory
@both
@pytest.mark.parametrize("window, second, group, dim", [(50, False, 1, 24), (16, True, 3, 24), (64, False, 9, 24), (129, True, 2, 72), (1, False, 1, 24)])
def test_window_edges(cuda, tmp_path, window, second, group, dim, f32):
    m = lm.window_needle(tmp_path, window, second, group, dim)
    d = driver(m, f32, max_seq=700)
    for key_at in (0, 1, 15, 16, 63, 64, 127, 190):
        # QUERY just before KEY (must not see it), right behind it, as the last position that sees it and as the first that does not
        at = sorted({p for p in (key_at - 1, key_at + 1, key_at + window - 1, key_at + window) if p >= 0 and p != key_at})
        tok = lm.needle_tokens(330, key_at, at, seed=key_at)
        tok[key_at] = lm.KEY
        want, bar = m.plain(tok)[0], m.bar(tok, f32)
        assert bar < (2e-4 if f32 else 0.3)
        edge = key_at + window
        for cuts in ([330], [edge, 330], [edge - 1, 1, 1, 2, 330], [key_at or 1, 2, 64], [max(1, edge - 40)] + [1] * 45 + [330]):
            d.release(0)
            err = lm.rel_error(run(d, 0, tok, [c for c in cuts if c > 0]), want)
            assert err.max() < bar, (key_at, cuts[:4], int(err.argmax()), err.max(), bar)
    d.close()


@both
@pytest.mark.parametrize("conv, dim", [(3, 20), (6, 140), (1, 20)])
def test_memory_far_back(cuda, tmp_path, conv, dim, f32):
    """What one token wrote into the state shows until the end, wherever the prompt is cut."""
    m = lm.memory_model(tmp_path, conv, dim)
    d = driver(m, f32)
    for key_at in (0, 1, 62, 63, 64, 130):
        tok = lm.needle_tokens(300, key_at, [], seed=key_at)
        check(m, d, tok, ([300], [key_at + 1, 300], [key_at or 1, 1, 63, 2], [key_at + 2, 16, 1, 80, 64], [100] + [1] * 200), f32)
    d.close()


@both
def test_repeated_writes_to_one_key(cuda, tmp_path, f32):
    """A run of one token: every write after the first few finds its key in the state already."""
    m = lm.memory_model(tmp_path)
    tok = lm.needle_tokens(150, list(range(20, 110)), [], seed=3)
    d = driver(m, f32)
    check(m, d, tok, ([150], [1], [50, 2, 64]), f32)
    d.close()


# ----------------------------------------------------------------------------------------------- slots, batches, decoding
@both
def test_slots_are_used_again(cuda, tmp_path, f32):
    m = lm.Model(tmp_path, lm.lanedra_mixed(), 10)
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
    m = lm.Model(tmp_path, lm.lanedra_mixed(), 12)
    seqs = [tokens_for(m, n, 20 + n) for n in (90, 33, 140)]
    d = driver(m, f32, batch=3, max_portion=30)
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
    m = lm.Model(tmp_path, lm.lanedra_mixed(), 13)
    tok = tokens_for(m, 330, 6)
    d = driver(m, f32, max_portion=32)
    err = lm.rel_error(run(d, 0, tok, [30] + [1] * 300), m.plain(tok)[0])
    assert err.max() < m.bar(tok, f32) and err[300:].mean() < 3 * err[:60].mean() + 1e-6
    d.close()


@pytest.mark.parametrize("batch, graph", [(1, True), (3, False), (11, True), (20, True)])
def test_greedy_generation_matches_plain(cuda, tmp_path, batch, graph):
    """32-bit greedy generation of unequal prompts through begin / step / result: the ids of the plain evaluation."""
    m = lm.Model(tmp_path, lm.lanedra_mixed(), 14)
    lens = [1, 37, 2, 90, 5, 64, 65, 3, 16, 17, 33, 8, 1, 120, 50, 4, 6, 7, 9, 10][:batch]
    prompts = [tokens_for(m, n, 100 + i).tolist() for i, n in enumerate(lens)]
    d = driver(m, True, batch=batch, max_seq=160, max_prompt=130, max_new=8, use_graph=graph, max_portion=50)
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

    m = lm.Model(tmp_path, lm.lanedra_mixed(), 15)
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


# ----------------------------------------------------------------------------------------------- C entry points
class Rows(C.Structure):
    _fields_ = [("T", C.c_int), ("row_slot", C.c_void_p), ("row_pos", C.c_void_p), ("slot", C.c_int), ("pos0", C.c_int)]


class DiffArgs(C.Structure):
    _fields_ = ([(n, C.c_int) for n in ("heads", "kv_heads", "dim", "V", "window", "rot_dims")] + [("cs", C.c_void_p), ("max_seq", C.c_int)] +
                [(n, C.c_float) for n in ("scale", "lam", "out_scale", "eps")] + [("cache", C.c_void_p), ("cap", C.c_int), ("slots", C.c_int), ("q", C.c_void_p),
                ("k", C.c_void_p), ("v", C.c_void_p), ("ld", C.c_long), ("out", C.c_void_p), ("ldout", C.c_long), ("splits", C.c_int)])


@pytest.mark.parametrize("splits", [1, 2, 4, 8])
@pytest.mark.parametrize("window, cap, positions", [(0, 600, [0, 15, 16, 511, 599]), (200, 208, [1, 199, 200, 207, 208, 598]), (37, 48, [36, 37, 47, 48, 49, 597])])
def test_decode_attention_splits(cuda, window, cap, positions, splits):
    """One token per sequence against the plain formulas for every number of context splits, full and ring caches."""
    import torch
    from blackwell_b200 import _lib

    H, G, D, V, rot, max_seq, lam = 6, 2, 32, 40, 16, 600, 0.37
    rng = np.random.default_rng(window)
    B = len(positions)
    freq, gain = plain.yarn_frequencies(rot, 300.0, lm.yarn(5.0, 100.0, 8.0, 1.0))
    keys, values = lm.to_bf16(rng.standard_normal((B, max_seq, G, 2, D)))[1].reshape(B, max_seq, G, 2, D), rng.standard_normal((B, max_seq, G, V))
    values = lm.to_bf16(values)[1].reshape(values.shape)
    q = lm.to_bf16(rng.standard_normal((B, H, 2, D)) * 2)[1].reshape(B, H, 2, D)
    cache = torch.full((B, cap, G * (2 * D + V)), float("nan"), dtype=torch.bfloat16)
    proj = np.zeros((B, H * 2 * D + G * 2 * D + G * V))
    want = np.zeros((B, H, V))
    for b, p in enumerate(positions):
        rotated = plain.rotate_half(keys[b], np.arange(max_seq), rot, freq, gain)
        rotated = lm.to_bf16(rotated)[1].reshape(rotated.shape)
        lo = max(0, p - window + 1) if window else 0
        for j in range(lo, p):
            cache[b, j % cap] = torch.from_numpy(np.concatenate([rotated[j].reshape(G, 2 * D), values[b, j]], 1).reshape(-1))
        proj[b] = np.concatenate([q[b].ravel(), keys[b, p].ravel(), values[b, p].ravel()])
        qr = plain.rotate_half(q[b][None], [p], rot, freq, gain)[0]
        for h in range(H):
            a = [plain.softmax(rotated[lo:p + 1, h // 3, i] @ qr[h, i] * 0.2) @ values[b, lo:p + 1, h // 3] for i in range(2)]
            want[b, h] = plain.rms_unit(a[0] - lam * a[1], 1e-5) * 0.6
    cs = np.stack([np.cos(np.arange(max_seq)[:, None] * freq) * gain, np.sin(np.arange(max_seq)[:, None] * freq) * gain], -1)
    dev = {n: t.cuda() for n, t in dict(cache=cache, proj=torch.from_numpy(proj).to(torch.bfloat16), cs=torch.from_numpy(cs).float(),
                                        slot=torch.arange(B, dtype=torch.int32), pos=torch.tensor(positions, dtype=torch.int32)).items()}
    out = torch.zeros((B, H * V), dtype=torch.bfloat16, device="cuda")
    pp = dev["proj"].data_ptr()
    a = DiffArgs(H, G, D, V, window, rot, dev["cs"].data_ptr(), max_seq, 0.2, lam, 0.6, 1e-5, dev["cache"].data_ptr(), cap, B, pp, pp + 2 * H * 2 * D,
                 pp + 2 * (H + G) * 2 * D, proj.shape[1], out.data_ptr(), H * V, splits)
    r = Rows(B, dev["slot"].data_ptr(), dev["pos"].data_ptr(), 0, 0)
    assert _lib.load().bw_diff_attention(C.byref(a), C.byref(r), 0, None) == 0
    torch.cuda.synchronize()
    got = out.float().cpu().numpy().reshape(want.shape)
    assert np.isfinite(got).all() and np.abs(got - want).max() < 0.02 * np.abs(want).max()
    for b, p in enumerate(positions):   # the new row is in the cache
        new = np.concatenate([plain.rotate_half(keys[b, p][None], [p], rot, freq, gain)[0].reshape(G, 2 * D), values[b, p]], 1).reshape(-1)
        assert np.abs(dev["cache"][b, p % cap].float().cpu().numpy() - new).max() < 0.02 * np.abs(new).max()


def test_rejected_calls(cuda, tmp_path):
    from blackwell_b200 import _lib
    from blackwell_b200.kernels import KernelError

    L = _lib.load()
    one = C.c_void_p(16)
    good = dict(heads=4, kv_heads=2, dim=16, V=16, window=8, rot_dims=8, cs=one, max_seq=64, scale=1.0, lam=0.1, out_scale=1.0, eps=1e-5, cache=one,
                cap=64, slots=1, q=one, k=one, v=one, ld=64, out=one, ldout=64, splits=1)
    for change in (dict(kv_heads=3), dict(rot_dims=18), dict(rot_dims=7), dict(cap=6), dict(cap=40), dict(slots=0), dict(ld=63), dict(V=4000), dict(v=None), dict(window=-1)):
        assert L.bw_diff_attention(C.byref(DiffArgs(**{**good, **change})), C.byref(Rows(2, None, None, 0, 0)), 0, None) != 0, change
    m = lm.Model(tmp_path, lm.lanedra_mixed(), 16)
    cfg = json.loads(json.dumps(m.cfg))
    cfg["layers"][0]["mixer"]["vdim"] = 36      # sizes that the weights do not have
    cfg["layers"][2]["mixer"]["vdim"] = cfg["layers"][5]["mixer"]["vdim"] = 36
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(KernelError):
        driver(m, False)


# ----------------------------------------------------------------------------------------------- programs
def test_daemon_generates_from_ids(cuda, tmp_path):
    m = lm.Model(tmp_path / "m", lm.lanedra_mixed(), 17)
    prompts = [tokens_for(m, n, 300 + n).tolist() for n in (5, 40, 1)]
    exe = os.path.join(ROOT, "blackwell_b200", "lib", "inference_server_w4a8")
    p = subprocess.run([exe, "--weights", m.dir, "--batch", "2", "--max-seq", "128", "--dtype", "float32"],
                       input=json.dumps({"prompt_ids": prompts, "max_tokens": 4}) + "\n", capture_output=True, text=True, timeout=120)
    assert p.returncode == 0, p.stderr[-2000:]
    for got, prompt in zip(json.loads(p.stdout.splitlines()[0])["tokens"], prompts):
        assert got == m.greedy(prompt, 5)


@both
def test_trace_runner(cuda, tmp_path, f32):
    m = lm.Model(tmp_path / "m", lm.lanedra_mixed(), 18)
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
    for i, want in rows.items():
        got = np.fromfile(out / f"{i}.f32", "<f4").reshape(want.shape)
        assert lm.rel_error(got, want).max() < m.bar(a, f32)
