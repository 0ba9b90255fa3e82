"""Parity of the quantizers, RMSNorm / SwiGLU / residual kernels, KV update, GQA decode attention and greedy
sampling (through the C ABI) against the CPU oracle, and against the reference's own CUDA kernels where those
are valid."""
import numpy as np
import pytest

import oracle
from blackwell_b200 import synth
from tests.util import max_abs_rel, to_dev

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def k(cuda):
    from blackwell_b200 import kernels

    return kernels


def _edge_activations(M, K, seed):
    x = synth.activations_f16(M, K, seed).astype(np.float32)
    x[0, :16] = 0.0                  # all-zero block
    x[0, 16:32] = 3e-11              # below both degenerate thresholds
    if K >= 64:
        x[-1, 32:48] = 1000.0        # equal magnitudes: every element hits the clamp
        x[-1, 48] = -7.5 * (np.abs(x[-1, 48:64]).max() / 7)  # a value beyond the block's own range
    return x


@pytest.mark.parametrize("M,K", [(1, 4096), (8, 10944), (3, 48), (64, 5120)])
def test_quantize_int4_bit_exact(k, M, K):
    import torch

    x = _edge_activations(M, K, 100 + M)
    q = torch.empty((M, K // 2), dtype=torch.uint8, device="cuda")
    s = torch.empty((M, K // 16), dtype=torch.float32, device="cuda")
    if M == 1:
        k.quantize_int4(q, s, to_dev(x), K)
    else:
        k.quantize_int4_batched(q, s, to_dev(x), K, M)
    qr, sr = oracle.quantize_int4(x)
    assert np.array_equal(q.cpu().numpy(), qr) and np.array_equal(s.cpu().numpy(), sr)


@pytest.mark.parametrize("M,K", [(1, 4096), (8, 10944), (2, 32)])
def test_quantize_int8_bit_exact(k, M, K):
    import torch

    x = _edge_activations(M, K, 110 + M)
    q = torch.empty((M, K), dtype=torch.int8, device="cuda")
    s = torch.empty((M, K // 16), dtype=torch.float32, device="cuda")
    k.quantize_int8(q, s, to_dev(x), M * K)
    qr, sr = oracle.quantize_int8(x)
    assert np.array_equal(q.cpu().numpy(), qr) and np.array_equal(s.cpu().numpy(), sr)
    # binary16 input variant: same bits as quantizing the widened values
    x16 = x.astype(np.float16)
    k.quantize_int8_f16(q, s, to_dev(x16.view(np.uint16)), M * K)
    qr, sr = oracle.quantize_int8(x16.astype(np.float32))
    assert np.array_equal(q.cpu().numpy(), qr) and np.array_equal(s.cpu().numpy(), sr)


def test_quantizers_match_reference_cuda(k):
    import torch

    from oracle import ref_cuda

    if not ref_cuda.available():
        pytest.skip("oracle/_ref/libblackwell_ref.so is not built (`make -C oracle ref` needs the reference sources)")

    M, K = 4, 4096
    x = to_dev(_edge_activations(M, K, 120))
    q = torch.empty((M, K // 2), dtype=torch.uint8, device="cuda")
    s = torch.empty((M, K // 16), dtype=torch.float32, device="cuda")
    qr, sr = torch.empty_like(q), torch.empty_like(s)
    k.quantize_int4_batched(q, s, x, K, M)
    ref_cuda.quantize_int4_batched(qr, sr, x, K, M)
    assert torch.equal(q, qr) and torch.equal(s, sr)
    q8 = torch.empty((M, K), dtype=torch.int8, device="cuda")
    s8 = torch.empty((M * K // 16,), dtype=torch.float32, device="cuda")
    q8r, s8r = torch.empty_like(q8), torch.empty_like(s8)
    k.quantize_int8(q8, s8, x, M * K)
    ref_cuda.quantize_int8(q8r, s8r, x, M * K)
    assert torch.equal(q8, q8r) and torch.equal(s8, s8r)


@pytest.mark.parametrize("M,H", [(1, 4096), (8, 4096), (3, 5120), (2, 10944), (1, 100)])
def test_rmsnorm(k, M, H):
    import torch

    x = synth.activations_f16(M, H, 130).astype(np.float32)
    w = synth.norm_weight(H, 131)
    out = torch.empty((M, H), dtype=torch.float32, device="cuda")
    if M == 1:
        k.fused_rmsnorm(out, to_dev(x), to_dev(w), H, 1e-6)
    else:
        k.fused_rmsnorm_batched(out, to_dev(x), to_dev(w), H, 1e-6, M)
    ref = oracle.rmsnorm(x, w)
    assert np.allclose(out.cpu().numpy(), ref, rtol=2e-6, atol=1e-7)


def test_rmsnorm_matches_reference_cuda_within_its_limit(k):
    import torch

    from oracle import ref_cuda

    if not ref_cuda.available():
        pytest.skip("oracle/_ref/libblackwell_ref.so is not built (`make -C oracle ref` needs the reference sources)")

    M, H = 4, 4096
    x, w = to_dev(synth.activations_f16(M, H, 132).astype(np.float32)), to_dev(synth.norm_weight(H, 133))
    a, b = torch.empty_like(x), torch.empty_like(x)
    k.fused_rmsnorm_batched(a, x, w, H, 1e-6, M)
    ref_cuda.fused_rmsnorm_batched(b, x, w, H, 1e-6, M)
    assert torch.allclose(a, b, rtol=2e-6, atol=1e-7)


@pytest.mark.parametrize("n", [10944, 4096, 7, 1025])
def test_swiglu_and_vector_add(k, n):
    import torch

    g = synth.activations_f16(1, n if n % 16 == 0 else 16 * (n // 16 + 1), 140).astype(np.float32)[0, :n] * 4
    u = synth.activations_f16(1, n if n % 16 == 0 else 16 * (n // 16 + 1), 141).astype(np.float32)[0, :n]
    out = torch.empty(n, dtype=torch.float32, device="cuda")
    k.apply_swiglu(out, to_dev(g), to_dev(u), n)
    assert np.allclose(out.cpu().numpy(), oracle.swiglu(g, u), rtol=2e-6, atol=1e-7)
    gd = to_dev(g)
    k.apply_swiglu(gd, gd, to_dev(u), n)  # in place, as the decode loop calls it
    assert np.allclose(gd.cpu().numpy(), oracle.swiglu(g, u), rtol=2e-6, atol=1e-7)
    k.vector_add_fp32(out, to_dev(g), to_dev(u), n)
    assert np.array_equal(out.cpu().numpy(), oracle.vector_add(g, u))


@pytest.mark.parametrize("N", [4096, 10944, 5120])
def test_fused_quant_int4_variants(k, N):
    """fused_rmsnorm_quant_int4 / fused_swiglu_quant_int4 (scale floor 1e-9, clamp +-7).  The activation they
    quantize differs from the CPU's in the last bit, which can move a value across a rounding tie: scales
    must agree to 1e-6 relative and at most 0.1% of the nibbles may differ, each by one step."""
    import torch

    x = synth.activations_f16(1, N, 150).astype(np.float32)[0]
    u = synth.activations_f16(1, N, 151).astype(np.float32)[0]
    w = synth.norm_weight(N, 152)
    q = torch.empty(N // 2, dtype=torch.uint8, device="cuda")
    s = torch.empty(N // 16, dtype=torch.float32, device="cuda")

    def check(ref_act):
        qr, sr = oracle.quantize_int4_fusedrule(ref_act)
        assert np.allclose(s.cpu().numpy(), sr, rtol=1e-6)
        a, b = q.cpu().numpy(), qr
        lo = np.abs((a & 15).astype(int) - (b & 15).astype(int))
        hi = np.abs((a >> 4).astype(int) - (b >> 4).astype(int))
        assert max(lo.max(), hi.max()) <= 1
        assert (lo != 0).sum() + (hi != 0).sum() <= max(1, N // 1000)

    k.fused_rmsnorm_quant_int4(q, s, to_dev(x), to_dev(w), N, 1e-6)
    check(oracle.rmsnorm(x, w))
    k.fused_swiglu_quant_int4(q, s, to_dev(x), to_dev(u), N)
    check(oracle.swiglu_fusedform(x, u))


def test_rope_decode(k):
    import torch

    heads, hd, max_seq, pos = 8, 128, 64, 37
    d = synth.rng(160).normal(size=heads * hd).astype(np.float32)
    i = np.arange(hd // 2)
    t = np.arange(max_seq)[:, None] * np.power(1e6, -2.0 * i / hd)[None]
    cos, sin = np.cos(t).astype(np.float32), np.sin(t).astype(np.float32)
    dd = to_dev(d)
    k.fused_rope_decode(dd, to_dev(cos), to_dev(sin), to_dev(np.array([pos], np.int32)), heads, hd, max_seq)
    p = d.reshape(heads, hd // 2, 2)
    ref = np.stack([p[..., 0] * cos[pos] - p[..., 1] * sin[pos], p[..., 0] * sin[pos] + p[..., 1] * cos[pos]], -1)
    assert np.allclose(dd.cpu().numpy().reshape(heads, hd // 2, 2), ref, rtol=1e-6, atol=1e-6)


def test_update_kv_cache(k):
    import torch

    nh, hd, max_seq, pos = 8, 128, 32, 9
    kn = synth.rng(170).normal(size=nh * hd).astype(np.float32)
    vn = synth.rng(171).normal(size=nh * hd).astype(np.float32)
    kc = torch.zeros((nh, max_seq, hd), dtype=torch.float32, device="cuda")
    vc = torch.zeros_like(kc)
    k.update_kv_cache(kc, vc, to_dev(kn), to_dev(vn), 0, pos, nh, hd, max_seq)
    kr, vr = np.zeros((nh, max_seq, hd), np.float32), np.zeros((nh, max_seq, hd), np.float32)
    oracle.update_kv(kr, vr, kn, vn, pos, nh, hd, max_seq)
    assert np.array_equal(kc.cpu().numpy(), kr) and np.array_equal(vc.cpu().numpy(), vr)
    k.update_kv_cache_device(kc, vc, to_dev(vn), to_dev(kn), 0, to_dev(np.array([pos + 1], np.int32)), nh, hd,
                             max_seq)
    oracle.update_kv(kr, vr, vn, kn, pos + 1, nh, hd, max_seq)
    assert np.array_equal(kc.cpu().numpy(), kr) and np.array_equal(vc.cpu().numpy(), vr)
    from blackwell_b200.kernels import KernelError

    with pytest.raises(KernelError):  # same contract as the reference: only batch_idx 0
        k.update_kv_cache(kc, vc, to_dev(kn), to_dev(vn), 1, pos, nh, hd, max_seq)


ATTN_CASES = [  # (M, nqh, nkv, max_seq, pos, layers, layer)
    (1, 32, 8, 256, 0, 1, 0), (1, 32, 8, 256, 1, 2, 1), (1, 32, 8, 4096, 2047, 1, 0), (2, 32, 8, 512, 300, 2, 1),
    (8, 32, 8, 2048, 2047, 1, 0), (1, 64, 8, 4200, 4100, 1, 0), (3, 8, 8, 128, 77, 1, 0), (2, 16, 8, 130, 129, 1, 0),
]


@pytest.mark.parametrize("M,nqh,nkv,max_seq,pos,layers,layer", ATTN_CASES)
def test_attention_decode_fp32_cache(k, M, nqh, nkv, max_seq, pos, layers, layer):
    import torch

    hd = 128
    g = synth.rng(180 + M + pos)
    Q = g.normal(size=(M, nqh * hd)).astype(np.float32)
    layer_elems = nkv * max_seq * hd
    kv_batch = layers * layer_elems
    Kc = g.normal(size=M * kv_batch).astype(np.float32)
    Vc = g.normal(size=M * kv_batch).astype(np.float32)
    out = torch.full((M, nqh * hd), float("nan"), dtype=torch.float32, device="cuda")
    Kd, Vd = to_dev(Kc), to_dev(Vc)
    k.attention_decode_batched_gqa(out, to_dev(Q), Kd, Vd, pos, nqh, nkv, hd, max_seq, M, kv_batch,
                                   layer * layer_elems)
    ref = oracle.attention_decode_gqa(Q, Kc, Vc, pos, nqh, nkv, hd, max_seq, M, kv_batch, layer * layer_elems)
    assert max_abs_rel(out.cpu().numpy(), ref) < 1e-4
    out2 = torch.empty_like(out)
    k.attention_decode_batched_gqa_device(out2, to_dev(Q), Kd, Vd, to_dev(np.array([pos], np.int32)), nqh, nkv, hd,
                                          max_seq, M, kv_batch, layer * layer_elems)
    assert max_abs_rel(out2.cpu().numpy(), ref) < 1e-4


def test_attention_matches_reference_cuda_short_context(k):
    import torch

    from oracle import ref_cuda

    if not ref_cuda.available():
        pytest.skip("oracle/_ref/libblackwell_ref.so is not built (`make -C oracle ref` needs the reference sources)")

    M, nqh, nkv, hd, max_seq, pos = 1, 32, 8, 128, 512, 200
    g = synth.rng(190)
    Q = to_dev(g.normal(size=(M, nqh * hd)).astype(np.float32))
    Kc = to_dev(g.normal(size=nkv * max_seq * hd).astype(np.float32))
    Vc = to_dev(g.normal(size=nkv * max_seq * hd).astype(np.float32))
    a, b = torch.empty_like(Q), torch.empty_like(Q)
    k.attention_decode_batched_gqa(a, Q, Kc, Vc, pos, nqh, nkv, hd, max_seq, M, nkv * max_seq * hd, 0)
    ref_cuda.attention_decode_batched_gqa(b, Q, Kc, Vc, pos, nqh, nkv, hd, max_seq, M, nkv * max_seq * hd, 0)
    torch.cuda.synchronize()
    ref = oracle.attention_decode_gqa(Q.cpu().numpy(), Kc.cpu().numpy(), Vc.cpu().numpy(), pos, nqh, nkv, hd,
                                      max_seq, M, nkv * max_seq * hd, 0)
    assert max_abs_rel(a.cpu().numpy(), ref) < 1e-4
    # the reference kernel's in-place softmax is racy; record how far it lands from the oracle rather than
    # requiring equality, but it must be in the same neighbourhood when the race does not bite
    print("reference attention vs oracle:", max_abs_rel(b.cpu().numpy(), ref))


def test_attention_arrival_counters_survive_a_smaller_call_before_a_larger_one(k):
    """The split kernels count arrivals in the library's scratch block.  A call with few (sequence, kv head) pairs
    followed by one with many once found the earlier call's partial records where it expected zeroed counters; the
    counters now own a fixed region."""
    import torch

    hd, max_seq = 128, 640
    k.set_tuning(22, 200)   # the split rule that aims at two CTAs per SM: these small contexts are then split
    try:
        _counter_cases(k, hd, max_seq)
    finally:
        k.set_tuning(22, 0)


def _counter_cases(k, hd, max_seq):
    import torch

    for M, nqh, nkv, seed in [(2, 32, 8, 240), (24, 32, 8, 241), (3, 16, 4, 242), (40, 8, 8, 243)]:
        g = synth.rng(seed)
        Q = g.normal(size=(M, nqh * hd)).astype(np.float32)
        Kc = synth.kv_cache_f16((M, nkv, max_seq, hd), seed + 10)
        Vc = synth.kv_cache_f16((M, nkv, max_seq, hd), seed + 20)
        pos = np.array([max_seq - 1 - 11 * (m % 9) for m in range(M)], np.int32)
        out = torch.full((M, nqh * hd), float("nan"), dtype=torch.float32, device="cuda")
        k.attention_decode_f16kv(out, to_dev(Q), to_dev(Kc.view(np.uint16)), to_dev(Vc.view(np.uint16)), to_dev(pos),
                                 max_seq, nqh, nkv, hd, max_seq, M, nkv * max_seq * hd, 0)
        ref = oracle.attention_decode_f16kv(Q, Kc, Vc, pos, nqh, nkv, hd, max_seq, M)
        assert max_abs_rel(out.cpu().numpy(), ref) < 1e-4, (M, nqh, nkv)


@pytest.mark.parametrize("nqh,nkv", [(32, 8), (4, 2)])
def test_attention_f16_cache_context_longer_than_the_hint(k, nqh, nkv):
    """The context hint only sizes the splits: sequences that have grown well past it (a captured step replayed many
    times) must still attend to every position (tensor-core kernel: 4 heads per kv head; scalar kernel: 2)."""
    import torch

    M, hd, max_seq, hint = 3, 128, 2048, 800   # three splits of 268 positions
    g = synth.rng(230)
    Q = g.normal(size=(M, nqh * hd)).astype(np.float32)
    Kc = synth.kv_cache_f16((M, nkv, max_seq, hd), 231)
    Vc = synth.kv_cache_f16((M, nkv, max_seq, hd), 232)
    pos = np.array([150, 1500, 2047], np.int32)
    out = torch.empty((M, nqh * hd), dtype=torch.float32, device="cuda")
    k.attention_decode_f16kv(out, to_dev(Q), to_dev(Kc.view(np.uint16)), to_dev(Vc.view(np.uint16)), to_dev(pos),
                             hint, nqh, nkv, hd, max_seq, M, nkv * max_seq * hd, 0)
    ref = oracle.attention_decode_f16kv(Q, Kc, Vc, pos, nqh, nkv, hd, max_seq, M)
    assert max_abs_rel(out.cpu().numpy(), ref) < 1e-4


@pytest.mark.parametrize("M,nqh,nkv,max_seq,ctx", [(1, 32, 8, 2048, 2048), (8, 32, 8, 2048, 2048),
                                                    (4, 64, 8, 4096, 4096), (2, 32, 8, 300, 131)])
def test_attention_decode_f16_cache_per_sequence_positions(k, M, nqh, nkv, max_seq, ctx):
    import torch

    hd = 128
    g = synth.rng(200 + M)
    Q = g.normal(size=(M, nqh * hd)).astype(np.float32)
    Kc = synth.kv_cache_f16((M, nkv, max_seq, hd), 201)
    Vc = synth.kv_cache_f16((M, nkv, max_seq, hd), 202)
    pos = np.array([ctx - 1 - 7 * m for m in range(M)], np.int32)
    out = torch.empty((M, nqh * hd), dtype=torch.float32, device="cuda")
    k.attention_decode_f16kv(out, to_dev(Q), to_dev(Kc.view(np.uint16)), to_dev(Vc.view(np.uint16)), to_dev(pos),
                             ctx, nqh, nkv, hd, max_seq, M, nkv * max_seq * hd, 0)
    ref = oracle.attention_decode_f16kv(Q, Kc, Vc, pos, nqh, nkv, hd, max_seq, M)
    assert max_abs_rel(out.cpu().numpy(), ref) < 1e-4


@pytest.mark.parametrize("V", [151643, 1000, 7, 151936])
def test_argmax_and_penalty(k, V):
    import torch

    logits = synth.rng(210 + V).normal(size=V).astype(np.float32)
    logits[V // 2] = logits.max()  # an exact tie: lowest index wins
    ld = to_dev(logits)
    out = torch.zeros(1, dtype=torch.int32, device="cuda")
    k.sample_argmax_gpu(ld, V, out)
    assert int(out.item()) == oracle.argmax(logits)
    k.sample_gpu(ld, V, 0.0, 0, out, 1234, 0)
    assert int(out.item()) == oracle.argmax(logits)
    k.sample_argmax_gpu(ld, V, out)  # second call: the static ticket was reset
    assert int(out.item()) == oracle.argmax(logits)
    recent = np.array([0, V - 1, V // 2, 0], np.int32)
    k.apply_repetition_penalty(ld, to_dev(recent), recent.size, 1.3, V)
    assert np.array_equal(ld.cpu().numpy(), oracle.repetition_penalty(logits, recent, 1.3))


def test_temperature_sampling_follows_softmax_topk(k):
    import torch

    V, top_k = 1000, 5
    logits = synth.rng(220).normal(size=V).astype(np.float32) * 3
    ld = to_dev(logits)
    out = torch.zeros(1, dtype=torch.int32, device="cuda")
    keep = set(np.argsort(-logits)[:top_k].tolist())
    counts = {}
    for step in range(300):
        k.sample_gpu(ld, V, 0.8, top_k, out, 42, step)
        t = int(out.item())
        assert t in keep
        counts[t] = counts.get(t, 0) + 1
    p = np.exp(logits - logits.max())
    idx = sorted(keep)
    pk = p[idx] / p[idx].sum()
    emp = np.array([counts.get(i, 0) for i in idx]) / 300.0
    assert np.abs(emp - pk).max() < 0.12
    assert np.array_equal(ld.cpu().numpy(), logits)  # the logits are left intact
