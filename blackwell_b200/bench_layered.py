"""Throughput of the config.json models with the layer sizes of a real model (random weights), beside another model of the
same width, and the time of each kernel against its roofline.  Run through ``bench.py --layered``."""
from __future__ import annotations

import ctypes as C
import shutil
import tempfile

import numpy as np
import torch

from . import _lib, synth

L = _lib.load()


class Rows(C.Structure):
    _fields_ = [("T", C.c_int), ("row_slot", C.c_void_p), ("row_pos", C.c_void_p), ("slot", C.c_int), ("pos0", C.c_int)]


class RecurrenceArgs(C.Structure):
    _fields_ = ([(n, C.c_void_p) for n in ("q", "k", "v")] + [(n, C.c_long) for n in ("ldq", "ldk", "ldv")] +
                [(n, C.c_int) for n in ("heads", "N", "V", "groups")] +
                [(n, C.c_void_p) for n in ("log_decay", "weight", "head_log_decay")] + [("const_weight", C.c_float)] +
                [(n, C.c_void_p) for n in ("D", "S", "o")] + [("ldo", C.c_long)])


class DiffArgs(C.Structure):
    _fields_ = ([(n, C.c_int) for n in ("heads", "kv_heads", "dim", "V", "window", "rot_dims")] + [("cs", C.c_void_p), ("max_seq", C.c_int)] +
                [(n, C.c_float) for n in ("scale", "lam", "out_scale", "eps")] + [("cache", C.c_void_p), ("cap", C.c_int), ("slots", C.c_int), ("q", C.c_void_p),
                ("k", C.c_void_p), ("v", C.c_void_p), ("ld", C.c_long), ("out", C.c_void_p), ("ldout", C.c_long), ("splits", C.c_int)])


L.bw_delta_rule_scratch_bytes.restype = C.c_size_t


class LatentArgs(C.Structure):
    _fields_ = ([(n, C.c_int) for n in ("heads", "dim", "rot", "V", "R", "rot_dims")] + [("scale", C.c_float), ("eps", C.c_float),
                ("cs", C.c_void_p), ("max_seq", C.c_int), ("cache", C.c_void_p), ("ldc", C.c_long), ("q", C.c_void_p), ("ldq", C.c_long),
                ("dkv", C.c_void_p), ("gate", C.c_void_p), ("ld32", C.c_long), ("dkv_norm", C.c_void_p), ("Wkv", C.c_void_p),
                ("ldw", C.c_long), ("sink", C.c_void_p), ("out", C.c_void_p), ("ldout", C.c_long), ("qabs", C.c_void_p),
                ("part", C.c_void_p), ("splits", C.c_int), ("kv", C.c_void_p)])


def _stream():
    return C.c_void_p(torch.cuda.current_stream().cuda_stream)


def _ok(e):
    if e != 0:
        raise RuntimeError(f"kernel call failed: {e}")


def linear(y, x, W, T, N, K, y_f32=0, epi=0):
    _ok(L.bw_linear_bf16(C.c_void_p(y.data_ptr()), C.c_long(y.stride(0)), C.c_void_p(x.data_ptr()), C.c_long(x.stride(0)),
                         C.c_void_p(W.data_ptr()), C.c_long(W.stride(0)), T, N, K, y_f32, 0, epi, C.c_float(0), _stream()))


def graph_us(run, reps, rounds=5):
    """Median over the rounds of the time per call of run(i), i = 0 .. reps - 1, captured in one CUDA graph."""
    for i in range(min(reps, 3)):
        run(i)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for i in range(reps):
            run(i)
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    ts = []
    for r in range(rounds + 3):
        e0.record()
        g.replay()
        e1.record()
        torch.cuda.synchronize()
        if r >= 3:
            ts.append(e0.elapsed_time(e1) / reps * 1e3)
    return float(np.median(ts))


COLD = 300 << 20   # rotate over more than this many bytes between uses of a buffer (L2: 126 MB)


def linear_records(peak, bf16_peak, cfg, rows=(1, 8, 32, 64, 256, 4096)):
    W, ff = cfg["width"], cfg["layers"][0]["mlp"]["ff"]
    mats = []
    for i in (0, 1, 3) if cfg["architecture"] == "Vifivik" else (0, 1, 2):
        m, t = cfg["layers"][i]["mixer"], cfg["layers"][i]["type"]
        H = m["heads"]
        n_in = {"mamba2": lambda: 2 * H * m["vdim"] + 2 * m["groups"] * m["state"] + H,
                "latent_attention": lambda: H * (m["dim"] + m["rot_dim"] + 1) + m["kv_rank"] + m["rot_dim"],
                "retention": lambda: 2 * H * (m["dim"] + m["vdim"]),
                "delta": lambda: 2 * H * (m["vdim"] + 1) + 2 * m["kv_heads"] * m["dim"],
                "attention": lambda: 2 * H * m["dim"] + (0 if "kv_from" in m else m["kv_heads"] * (2 * m["dim"] + m["vdim"]))}[t]()
        if "kv_from" in m:
            t += " on another cache"
        mats += [(t + " in", n_in, W, 0), (t + " out", W, H * m["vdim"], 0)]
    mats += [("gate+up", 2 * ff, W, 1), ("down", W, ff, 0), ("head", cfg["vocab"], W, 0)]
    out = []
    for T in rows:
        for name, N, K, epi in mats:
            if name == "head" and T > 64:
                continue
            copies = max(1, min(40, -(-COLD // (N * K * 2))))
            w = torch.randn((copies, N, K), device="cuda", dtype=torch.bfloat16) * K ** -0.5
            x = torch.randn((T, K), device="cuda", dtype=torch.bfloat16)
            cols = N // 2 if epi else N
            y32 = name.endswith("out") or name in ("down", "head")
            y = torch.empty((T, cols), device="cuda", dtype=torch.float32 if y32 else torch.bfloat16)
            us = graph_us(lambda i: linear(y, x, w[i % copies], T, N, K, int(y32), epi), max(copies, 12 if T < 4096 else 4))
            nbytes = N * K * 2 + T * K * 2 + T * cols * y.element_size()
            fl = 2.0 * T * N * K
            bound = max(nbytes / peak / 1e3, fl / bf16_peak / 1e6)   # us
            out.append({"kernel": "linear", "matrix": name, "T": T, "N": N, "K": K, "us": round(us, 2), "gbs": round(nbytes / us / 1e3, 1),
                        "tflops": round(fl / us / 1e6, 1), "roofline_frac": round(bound / us, 3)})
            del w
    torch.cuda.empty_cache()
    return out


def recurrence_records(peak, bf16_peak, cfg):
    """Mamba2 and retention (Vifivik) or the delta rule (Lanedra)."""
    out = []
    for i in (0, 3) if cfg["architecture"] == "Vifivik" else (0,):
        m, t = cfg["layers"][i]["mixer"], cfg["layers"][i]["type"]
        H, V = m["heads"], m["vdim"]
        N, G = (m["state"], m["groups"]) if t == "mamba2" else (m["dim"], m.get("kv_heads", H))
        for M, chunked in ((1, 0), (8, 0), (64, 0), (512, 1), (4096, 1)):
            slots = 1 if chunked else max(M, -(-COLD // (H * N * V * 4)) // M * M)
            S = torch.zeros((slots, H, N, V), device="cuda")
            q, k = (torch.randn((M, G * N), device="cuda", dtype=torch.bfloat16) for _ in range(2))
            v = torch.randn((M, H * V), device="cuda", dtype=torch.bfloat16)
            o = torch.empty((M, H * V), device="cuda")
            ld = torch.full((M, H), -0.02, device="cuda")
            w = torch.full((M, H), 0.05, device="cuda")
            ids = torch.arange(slots, device="cuda", dtype=torch.int32)
            pos = torch.full((slots,), 5, device="cuda", dtype=torch.int32)
            a = RecurrenceArgs(q.data_ptr(), k.data_ptr(), v.data_ptr(), G * N, G * N, H * V, H, N, V, G, ld.data_ptr(), w.data_ptr(), None, 0.0,
                               None, S.data_ptr(), o.data_ptr(), H * V)
            scratch = torch.empty(L.bw_delta_rule_scratch_bytes(M, H), device="cuda", dtype=torch.uint8)

            def run(j):
                r = Rows(M, None, None, 0, 5) if chunked else Rows(M, ids.data_ptr() + 4 * (j * M % slots), pos.data_ptr(), 0, 0)
                if t == "delta":
                    return _ok(L.bw_delta_rule(C.byref(a), C.c_float(1e-6), C.c_float(N ** -0.5), C.c_void_p(scratch.data_ptr()), C.byref(r),
                                               chunked, 0, _stream()))
                _ok(L.bw_linear_recurrence(C.byref(a), C.byref(r), chunked, 0, _stream()))

            us = graph_us(run, 4 if chunked else max(8, slots // M))
            if chunked:
                nbytes = M * (2 * G * N * 2 + H * V * 6)
                fl = 2.0 * M * H * (64 * (N + V) + 3 * N * V if t == "delta" else 64 * (N + V) / 2 + 2 * N * V)
            else:
                nbytes, fl = 2 * M * H * N * V * 4, 0.0
            bound = max(nbytes / peak / 1e3, fl / bf16_peak / 1e6)
            out.append({"kernel": "recurrence " + ("chunk" if chunked else "step"), "layer": t, "T": M, "us": round(us, 2),
                        "gbs": round(nbytes / us / 1e3, 1), "tflops": round(fl / us / 1e6, 1), "roofline_frac": round(bound / us, 3)})
            del S
    torch.cuda.empty_cache()
    return out


def diff_records(peak, bf16_peak, cfg):
    """Differential attention: token steps (context, window) and whole prompts."""
    m = cfg["layers"][1]["mixer"]
    H, G, D, V, rot = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]["dims"]
    seg, out = 2 * D + V, []
    for M, ctx, window, prompt in ((1, 4096, 0, 0), (8, 4096, 0, 0), (64, 4096, 0, 0), (1, 32768, 0, 0), (1, 4096, 1024, 0), (8, 4096, 1024, 0),
                                   (64, 4096, 1024, 0), (512, 512, 0, 1), (4096, 4096, 0, 1), (4096, 4096, 1024, 1)):
        see = min(ctx, window or ctx)
        cap = ctx if prompt else see
        slots = 1 if prompt else max(M, min(512, -(-COLD // (cap * G * seg * 2)) // M * M))
        cache = torch.randn((slots, cap, G * seg), device="cuda", dtype=torch.bfloat16)
        proj = torch.randn((M, H * 2 * D + G * seg), device="cuda", dtype=torch.bfloat16)
        cs = torch.ones((ctx, rot // 2, 2), device="cuda") * 0.7
        o = torch.empty((M, H * V), device="cuda", dtype=torch.bfloat16)
        ids = torch.arange(slots, device="cuda", dtype=torch.int32)
        pos = torch.full((slots,), ctx - 1, device="cuda", dtype=torch.int32)
        pp = proj.data_ptr()
        a = DiffArgs(H, G, D, V, window, rot, cs.data_ptr(), ctx, m["scale"], 0.5, 0.5, 1e-5, cache.data_ptr(), cap, slots, pp, pp + 2 * H * 2 * D,
                     pp + 2 * (H + G) * 2 * D, proj.stride(0), o.data_ptr(), H * V, 0)

        def run(j):
            r = Rows(M, None, None, 0, 0) if prompt else Rows(M, ids.data_ptr() + 4 * (j * M % slots), pos.data_ptr(), 0, 0)
            _ok(L.bw_diff_attention(C.byref(a), C.byref(r), 0, _stream()))

        us = graph_us(run, 4 if prompt else max(8, slots // M))
        pairs = M * see if not prompt else sum(min(i + 1, see) for i in range(M))
        nbytes = M * (H * (2 * D + V) + G * seg) * 2 + (0 if prompt else M * see * G * seg * 2)
        fl = 2.0 * pairs * H * 2 * (D + V)
        bound = max(nbytes / peak / 1e3, fl / bf16_peak / 1e6)
        out.append({"kernel": "differential attention " + ("prompt" if prompt else "decode"), "T": M, "ctx": ctx, "window": window, "us": round(us, 2),
                    "gbs": round(nbytes / us / 1e3, 1), "tflops": round(fl / us / 1e6, 1), "roofline_frac": round(bound / us, 3)})
        del cache
    torch.cuda.empty_cache()
    return out


def latent_records(peak, bf16_peak, cfg):
    m = cfg["layers"][1]["mixer"]
    H, dim, rot, R, V = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"], m["vdim"]
    D = R + rot
    out = []
    for M, ctx, expanded in ((1, 4096, 0), (8, 4096, 0), (64, 4096, 0), (1, 32768, 0), (512, 512, 1), (4096, 4096, 1)):
        slots = 1 if expanded else max(M, min(128, -(-COLD // (ctx * D * 2)) // M * M))
        cache = torch.randn((slots, ctx, D), device="cuda", dtype=torch.bfloat16)
        q = torch.randn((M, H * (dim + rot)), device="cuda", dtype=torch.bfloat16)
        f32 = torch.randn((M, D + H), device="cuda")
        nw, sink, cs = torch.ones(R, device="cuda"), torch.zeros(H, device="cuda"), torch.ones((ctx, rot // 2, 2), device="cuda") * 0.7
        wkv = torch.randn((H * (dim + V), R), device="cuda", dtype=torch.bfloat16) * R ** -0.5
        o = torch.empty((M, H * V), device="cuda", dtype=torch.bfloat16)
        splits = max(1, min(64, ctx // 64, 148 // (M * -(-H // 16))))
        rows = M if not expanded else 1
        qabs = torch.empty((rows * H * 2 * D,), device="cuda", dtype=torch.bfloat16)
        part = torch.empty((rows * H * splits * (R + 4),), device="cuda")
        kv = torch.empty((ctx if expanded else 1, H * (dim + V)), device="cuda", dtype=torch.bfloat16)
        ids = torch.arange(slots, device="cuda", dtype=torch.int32)
        pos = torch.full((slots,), ctx - 1, device="cuda", dtype=torch.int32)
        a = LatentArgs(H, dim, rot, V, R, rot, m["scale"], 1e-6, cs.data_ptr(), ctx, cache.data_ptr(), D, q.data_ptr(), q.stride(0),
                       f32.data_ptr(), f32.data_ptr() + 4 * D, D + H, nw.data_ptr(), wkv.data_ptr(), R, sink.data_ptr(), o.data_ptr(), H * V,
                       qabs.data_ptr(), part.data_ptr(), splits, kv.data_ptr())

        def run(j):
            r = Rows(M, None, None, 0, 0) if expanded else Rows(M, ids.data_ptr() + 4 * (j * M % slots), pos.data_ptr(), 0, 0)
            _ok(L.bw_latent_attention(C.byref(a), C.byref(r), expanded, 0, _stream()))

        us = graph_us(run, 4 if expanded else max(8, slots // M))
        if expanded:
            nbytes = wkv.numel() * 2 + M * (D * 2 + H * (dim + rot + V) * 2)
            fl = 2.0 * M * (M / 2) * H * (dim + rot + V) + 2.0 * M * H * (dim + V) * R
        else:
            nbytes = M * ctx * D * 2 + wkv.numel() * 2
            fl = 2.0 * M * H * (ctx * (D + R) + R * (dim + V))
        bound = max(nbytes / peak / 1e3, fl / bf16_peak / 1e6)
        out.append({"kernel": "latent attention " + ("expanded" if expanded else "absorbed"), "T": M, "ctx": ctx, "us": round(us, 2),
                    "gbs": round(nbytes / us / 1e3, 1), "tflops": round(fl / us / 1e6, 1), "roofline_frac": round(bound / us, 3)})
        del cache
    torch.cuda.empty_cache()
    return out


def model_records(peak, cfg, ctx=2048, prompt=4096, batches=(1, 8, 32, 64)):
    """Decode: one replay of the captured step per token, CUDA events, L2 flushed by the weights themselves (larger than
    L2).  Prefill: bw_decode_begin on one prompt, host to device copy of the ids included."""
    from .decode_driver import ModelDriver

    root = tempfile.mkdtemp()
    out = []
    try:
        weights = synth.write_random_model(root, cfg)
        state = cache = 0
        for l in cfg["layers"]:
            m = l["mixer"]
            if l["type"] == "latent_attention":
                cache += (m["kv_rank"] + m["rot_dim"]) * 2 * ctx
            elif l["type"] == "attention":
                cache += m["kv_heads"] * (2 * m["dim"] + m["vdim"]) * 2 * min(ctx, m["mask"]["size"])
            else:
                state += 8 * m["heads"] * m["vdim"] * (m["state"] if l["type"] == "mamba2" else m["dim"])
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        rng = np.random.default_rng(0)
        d = ModelDriver(root, batch=1, max_seq=prompt + 8, max_prompt=prompt + 1)
        for n in (512, prompt):
            ts = []
            for r in range(6):
                ids = [rng.integers(0, cfg["vocab"], n + 1).tolist()]
                torch.cuda.synchronize()
                e0.record()
                d.begin(ids)
                e1.record()
                torch.cuda.synchronize()
                ts.append(e0.elapsed_time(e1))
            ms = float(np.median(ts[3:]))
            fl = 2.0 * n * (weights / 2 - cfg["vocab"] * cfg["width"])
            out.append({"phase": "prefill", "tokens": n, "ms": round(ms, 3), "tok_s": round(n / ms * 1e3), "weight_tflops": round(fl / ms / 1e9, 1)})
        d.close()
        for b in batches:
            d = ModelDriver(root, batch=b, max_seq=ctx + 64, max_prompt=ctx, max_new=64)
            d.begin([rng.integers(0, cfg["vocab"], ctx).tolist() for _ in range(b)])
            ts = []
            for r in range(23):
                e0.record()
                d.step()
                e1.record()
                torch.cuda.synchronize()
                if r >= 3:
                    ts.append(e0.elapsed_time(e1))
            ms = float(np.median(ts))
            nbytes = weights + b * (state + cache)
            out.append({"phase": "decode", "batch": b, "ctx": ctx, "ms_per_step": round(ms, 4), "tok_s": round(b / ms * 1e3, 1), "bytes_per_step": nbytes,
                        "gbs": round(nbytes / ms / 1e6, 1), "roofline_frac": round(nbytes / ms / 1e6 / peak, 3)})
            d.close()
    finally:
        shutil.rmtree(root)
    return out
