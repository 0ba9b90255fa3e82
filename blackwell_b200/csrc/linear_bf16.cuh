// y = W x for bfloat16 weights.  Three kernels:
//   linear_stream_kernel  few rows of a small matrix: weights go straight from HBM to registers as the A operand of
//                         mma.sync -- the order of k inside a 32-wide block is permuted identically for both operands,
//                         which a dot product does not see, so that a thread's fragment is one 16-byte load -- and the
//                         activations sit in shared memory as the B operand.
//   linear_tc_kernel      tcgen05.mma kind::f16, weights as the 128-row operand, up to 256 rows of activations as the
//                         other, both through 128-byte-swizzled TMA.  Prompts: persistent CTAs, accumulators
//                         double-buffered in tensor memory.  Decode steps and short portions: the K range is split over a
//                         cluster of up to eight CTAs, two of which share an SM, and the partial sums are added through
//                         distributed shared memory in a fixed order.
//                         Both have their first weights in flight before they wait for the preceding kernel.
//   linear_f32_kernel     32-bit mode: fp32 activations, fp32 FMAs (the weights are bfloat16 values, exact in fp32).
#pragma once
#include <cuda.h>

#include "gemm_w4a8_tc.cuh"
#include "lm_device.cuh"
#include "lm_ops.h"

namespace bw {
namespace lm {

// Writes one finished output (column n of row t).
template <bool F32>
__device__ __forceinline__ void store_out(const LinearArgs& a, int t, int n, float v) {
    if (a.epi == kEpiSoftcap) v = a.softcap * tanhf(v / a.softcap);
    if (n >= a.split) {
        a.y32[(long)t * a.ldy32 + (n - a.split)] = v;
    } else if (F32 || a.y_f32) {
        static_cast<float*>(a.y)[(long)t * a.ldy + n] = v;
    } else {
        static_cast<bf16*>(a.y)[(long)t * a.ldy + n] = __float2bfloat16_rn(v);
    }
}

// ---------------------------------------------------------------------------------------------- up to 8 rows
constexpr int kStreamWarps = 8;
constexpr int kStreamU = 4;   // 32-wide k blocks per warp and load batch

__global__ void __launch_bounds__(kStreamWarps * 32) linear_stream_kernel(const LinearArgs a, int xs_stride) {
    extern __shared__ __align__(16) unsigned char smem[];
    float* red = reinterpret_cast<float*>(smem);                         // [warps][8][16]
    unsigned char* xs = smem + kStreamWarps * 8 * 16 * 4;                // [T][xs_stride] bytes
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, q = lane & 3;
    const int tiles = (a.N + 15) / 16, kw = (int)a.ldw;
    const int nkb = (kw + 31) / 32;
    const int iters = (nkb + kStreamWarps * kStreamU - 1) / (kStreamWarps * kStreamU);
    const uint4 zero4 = make_uint4(0, 0, 0, 0);
    auto load = [&](uint4 (&w)[kStreamU][2], int tile, int it) {
        const int r0 = tile * 16 + g, r1 = r0 + 8;
#pragma unroll
        for (int u = 0; u < kStreamU; ++u) {
            const int k = ((it * kStreamU + u) * kStreamWarps + warp) * 32 + q * 8;
            const bool ok = k < kw;
            w[u][0] = ok && r0 < a.N ? __ldcs(reinterpret_cast<const uint4*>(a.W + (long)r0 * a.ldw + k)) : zero4;
            w[u][1] = ok && r1 < a.N ? __ldcs(reinterpret_cast<const uint4*>(a.W + (long)r1 * a.ldw + k)) : zero4;
        }
    };
    uint4 cur[kStreamU][2], nxt[kStreamU][2];
    int tile = blockIdx.x;
    if (tile < tiles) load(cur, tile, 0);
    pdl_trigger();
    pdl_wait();
    // activations: columns >= K are zero; rows >= T are not stored (their fragments are zero registers)
    const int kpad = nkb * 32;
    const RowWalk walk(t, kStreamWarps * 32, kpad / 8);
    for (RowWalk w = walk; w.row < a.T; w.next()) {
        const int c = w.col * 8;
        uint4 v = zero4;
        if (c < a.K) {
            v = *reinterpret_cast<const uint4*>(static_cast<const bf16*>(a.x) + (long)w.row * a.ldx + c);
            if (c + 8 > a.K) {   // ragged end: keep only the real columns
                uint32_t* e = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    if (c + 2 * j >= a.K) e[j] = 0;
                    else if (c + 2 * j + 1 >= a.K) e[j] &= 0xFFFFu;
                }
            }
        }
        *reinterpret_cast<uint4*>(xs + (long)w.row * xs_stride + c * 2) = v;
    }
    __syncthreads();

    float acc[4] = {};
    int it = 0;
    while (tile < tiles) {
        int ntile = tile, nit = it + 1;
        if (nit == iters) { nit = 0; ntile += gridDim.x; }
        if (ntile < tiles) load(nxt, ntile, nit);
#pragma unroll
        for (int u = 0; u < kStreamU; ++u) {
            const int kb = (it * kStreamU + u) * kStreamWarps + warp;
            if (kb < nkb) {
                uint4 b = zero4;
                if (g < a.T) b = *reinterpret_cast<const uint4*>(xs + g * xs_stride + (kb * 32 + q * 8) * 2);
                mma_bf16(acc, cur[u][0].x, cur[u][1].x, cur[u][0].y, cur[u][1].y, b.x, b.y);
                mma_bf16(acc, cur[u][0].z, cur[u][1].z, cur[u][0].w, cur[u][1].w, b.z, b.w);
            }
        }
        if (nit == 0) {   // tile finished: add the warps' K shares
            float* p = red + warp * 8 * 16;
            p[(2 * q) * 16 + g] = acc[0];
            p[(2 * q + 1) * 16 + g] = acc[1];
            p[(2 * q) * 16 + g + 8] = acc[2];
            p[(2 * q + 1) * 16 + g + 8] = acc[3];
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[i] = 0.f;
            __syncthreads();
            if (a.epi == kEpiSwiglu) {
                if (t < 8 * 8) {
                    const int m = t >> 3, j = t & 7, n = tile * 16 + 2 * j;
                    float gt = 0.f, up = 0.f;
#pragma unroll
                    for (int w = 0; w < kStreamWarps; ++w) {
                        const float2 s = *reinterpret_cast<const float2*>(red + (w * 8 + m) * 16 + 2 * j);
                        gt += s.x;
                        up += s.y;
                    }
                    if (m < a.T && n < a.N)
                        static_cast<bf16*>(a.y)[(long)m * a.ldy + (n >> 1)] = __float2bfloat16_rn(silu_f(gt) * up);
                }
            } else {
                if (t < 8 * 16) {
                    const int m = t >> 4, n = tile * 16 + (t & 15);
                    float s = 0.f;
#pragma unroll
                    for (int w = 0; w < kStreamWarps; ++w) s += red[(w * 8 + m) * 16 + (t & 15)];
                    if (m < a.T && n < a.N) store_out<false>(a, m, n, s);
                }
            }
            __syncthreads();
        }
#pragma unroll
        for (int u = 0; u < kStreamU; ++u) { cur[u][0] = nxt[u][0]; cur[u][1] = nxt[u][1]; }
        tile = ntile;
        it = nit;
    }
}

// ---------------------------------------------------------------------------------------------- 32-bit mode
// 64 x 64 outputs per block of 256 threads, 16 k per step.
__global__ void __launch_bounds__(256) linear_f32_kernel(const LinearArgs a) {
    __shared__ float xs[16][68], ws[16][68];
    pdl_wait();
    const int t = threadIdx.x, n0 = blockIdx.x * 64, t0 = blockIdx.y * 64, ty = t >> 4, tx = t & 15;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < a.K; k0 += 16) {
        for (int i = t; i < 64 * 16; i += 256) {
            const int r = i >> 4, k = i & 15;
            xs[k][r] = t0 + r < a.T && k0 + k < a.K ? static_cast<const float*>(a.x)[(long)(t0 + r) * a.ldx + k0 + k] : 0.f;
            ws[k][r] = n0 + r < a.N && k0 + k < a.K ? to_f(a.W[(long)(n0 + r) * a.ldw + k0 + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            const float4 xv = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
            const float4 wv = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
            const float xr[4] = {xv.x, xv.y, xv.z, xv.w}, wr[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xr[i], wr[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = t0 + ty * 4 + i, n = n0 + tx * 4;
        if (r >= a.T) continue;
        if (a.epi == kEpiSwiglu) {
#pragma unroll
            for (int j = 0; j < 4; j += 2)
                if (n + j < a.N)
                    static_cast<float*>(a.y)[(long)r * a.ldy + ((n + j) >> 1)] = silu_f(acc[i][j]) * acc[i][j + 1];
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (n + j < a.N) store_out<true>(a, r, n + j, acc[i][j]);
        }
    }
}

// ---------------------------------------------------------------------------------------------- tcgen05
constexpr int kTcRows = 128;      // weight rows per tile (MMA M)
constexpr int kTcK = 64;          // k per stage: one 128-byte swizzle atom of bf16
constexpr int kTcThreads = 384;   // warp 0 copies, warp 1 MMAs, warps 4-11 epilogue (two per TMEM lane quarter)

__host__ __device__ constexpr int tc_stage_bytes(int NT) { return kTcRows * 128 + NT * 128; }
// split form: two CTAs share an SM; its accumulator tile for the cluster reduction, [NT][128] fp32, takes the place of the
// operand ring once the products are done
__host__ __device__ constexpr int tc_stages(int NT, bool split) { return split ? (NT >= 64 ? 4 : 5) : NT >= 256 ? 4 : NT >= 128 ? 6 : 8; }
__host__ __device__ constexpr int tc_smem_bytes(int NT, bool split) { return 1024 + 1024 + tc_stages(NT, split) * tc_stage_bytes(NT); }

// Shared-memory matrix descriptor: K-major rows of 128 bytes in the 128-byte swizzle, 8-row groups 1024 bytes apart.
__device__ __forceinline__ uint64_t desc_sw128(uint32_t addr) {
    return (uint64_t)((addr >> 4) & 0x3FFF) | (uint64_t)1 << 16 | (uint64_t)(1024 >> 4) << 32 | (uint64_t)1 << 46 | (uint64_t)2 << 61;
}
// Instruction descriptor: D fp32, A = B = bf16, both K-major, M = 128, N = n.
__host__ __device__ constexpr uint32_t idesc_bf16(int n) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(kTcRows >> 4) << 24);
}
__device__ __forceinline__ void tc_mma_f16(uint32_t tmem_d, uint64_t da, uint64_t db, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5}, p;\n\t}"
        ::"r"(tmem_d), "l"(da), "l"(db), "r"(idesc), "r"(accumulate), "r"(0u)
        : "memory");
}

// SPLIT: one tile per cluster of `ksplit` CTAs; otherwise persistent CTAs walk the tiles, weight rows fastest while the
// weights stay in L2, activation rows fastest when they do not (`ksplit` != 0 there).
template <int NT, bool SPLIT>
__global__ void __launch_bounds__(kTcThreads, SPLIT ? 2 : 1)
linear_tc_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x, const LinearArgs a,
                 int ksplit, int* status) {
    constexpr int S = tc_stages(NT, SPLIT), BYTES = tc_stage_bytes(NT), NACC = SPLIT ? 1 : 2;
    constexpr int COLS = SPLIT ? (NT < 32 ? 32 : NT) : 2 * NT;
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem);           // full[S], empty[S], dfull[2], dempty[2]
    volatile uint32_t* tmem_ptr = reinterpret_cast<volatile uint32_t*>(smem + 512);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + 520);
    unsigned char* stage0 = smem + 1024;
    float* part = reinterpret_cast<float*>(stage0);
    static_assert(!SPLIT || NT * kTcRows * 4 <= S * BYTES, "accumulator tile");
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31;
    auto full = [&](int i) { return smem_u32(&bars[i]); };
    auto empty = [&](int i) { return smem_u32(&bars[S + i]); };
    auto dfull = [&](int i) { return smem_u32(&bars[2 * S + i]); };
    auto dempty = [&](int i) { return smem_u32(&bars[2 * S + 2 + i]); };
    auto wait = [&](uint32_t bar, uint32_t parity) {
        if (mbar_try_wait(bar, parity)) return true;
        if (*abort_flag) return false;
        if (!mbar_wait(bar, parity)) { *abort_flag = 1; return false; }
        return true;
    };
    if (t == 0) {
        for (int i = 0; i < S; ++i) { mbar_init(full(i), 1); mbar_init(empty(i), 1); }
        for (int i = 0; i < 2; ++i) { mbar_init(dfull(i), 1); mbar_init(dempty(i), 8); }
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 1) {
        tc::tmem_alloc(smem_u32(smem + 512), COLS);
        tc::tmem_relinquish();
    }
    tc::tc_fence_before();
    __syncthreads();
    tc::tc_fence_after();
    const uint32_t tmem = *tmem_ptr;
    pdl_trigger();

    const int rtiles = (a.N + kTcRows - 1) / kTcRows, ttiles = (a.T + NT - 1) / NT, tiles = rtiles * ttiles;
    const bool tok_fast = !SPLIT && ksplit != 0;
    auto row_tile = [&](int tile) { return tok_fast ? tile / ttiles : tile % rtiles; };
    auto tok_tile = [&](int tile) { return tok_fast ? tile % ttiles : tile / rtiles; };
    const int nk = (a.K + kTcK - 1) / kTcK;
    const int kpart = SPLIT ? (int)(blockIdx.x % ksplit) : 0;
    const int kb0 = SPLIT ? (int)((long)nk * kpart / ksplit) : 0, kb1 = SPLIT ? (int)((long)nk * (kpart + 1) / ksplit) : nk;
    const int first = SPLIT ? (int)(blockIdx.x / ksplit) : (int)blockIdx.x;
    const int stride = SPLIT ? tiles : (int)gridDim.x;

    if (warp == 0) {
        if (lane == 0) {
            int n = 0;
            bool ok = true, waited = false;
            for (int tile = first; tile < tiles && ok; tile += stride) {
                const int row0 = row_tile(tile) * kTcRows, tok0 = tok_tile(tile) * NT;
                int kb = kb0;
                if (!waited) {   // weights do not depend on the kernel before: fill the ring with them first
                    const int pre = min(S, kb1 - kb0);
                    for (int i = 0; i < pre; ++i) {
                        mbar_expect_tx(full(i), BYTES);
                        tc::tma_load_2d(smem_u32(stage0 + i * BYTES), &map_w, (kb0 + i) * kTcK, row0, full(i));
                    }
                    pdl_wait();
                    for (int i = 0; i < pre; ++i)
                        tc::tma_load_2d(smem_u32(stage0 + i * BYTES + kTcRows * 128), &map_x, (kb0 + i) * kTcK, tok0, full(i));
                    waited = true;
                    n = pre;
                    kb += pre;
                }
                for (; kb < kb1; ++kb, ++n) {
                    const int s = n % S;
                    if (!wait(empty(s), ((n / S) & 1) ^ 1)) { ok = false; break; }
                    mbar_expect_tx(full(s), BYTES);
                    tc::tma_load_2d(smem_u32(stage0 + s * BYTES), &map_w, kb * kTcK, row0, full(s));
                    tc::tma_load_2d(smem_u32(stage0 + s * BYTES + kTcRows * 128), &map_x, kb * kTcK, tok0, full(s));
                }
            }
            if (!ok)   // copies still in flight land before the CTA leaves
                for (int i = max(0, n - S); i < n; ++i) mbar_wait(full(i % S), (i / S) & 1);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc = idesc_bf16(NT);
            int n = 0, w = 0;
            bool ok = true;
            for (int tile = first; tile < tiles && ok; tile += stride, ++w) {
                const int d = w % NACC;
                if (!wait(dempty(d), ((w / NACC) & 1) ^ 1)) { ok = false; break; }
                tc::tc_fence_after();
                for (int kb = kb0; kb < kb1; ++kb, ++n) {
                    const int s = n % S;
                    if (!wait(full(s), (n / S) & 1)) { ok = false; break; }
                    tc::tc_fence_after();
                    const uint64_t da = desc_sw128(smem_u32(stage0 + s * BYTES));
                    const uint64_t db = desc_sw128(smem_u32(stage0 + s * BYTES + kTcRows * 128));
#pragma unroll
                    for (int k = 0; k < kTcK / 16; ++k)   // 16 k = 32 bytes further inside the swizzle atom
                        tc_mma_f16(tmem + d * NT, da + 2 * k, db + 2 * k, idesc, kb > kb0 || k > 0);
                    tc::tc_commit(empty(s));
                }
                if (ok) tc::tc_commit(dfull(d));
            }
        }
    } else if (warp >= 4) {
        const int quarter = warp & 3, half = (warp - 4) >> 2;
        constexpr int CW = NT >= 64 ? 32 : 16;               // columns per read
        constexpr int HC = NT >= 32 ? NT / 2 : NT;           // columns per warp
        int w = 0;
        for (int tile = first; tile < tiles; tile += stride, ++w) {
            const int d = w % NACC;
            if (!wait(dfull(d), (w / NACC) & 1)) break;
            tc::tc_fence_after();
            const int row = row_tile(tile) * kTcRows + quarter * 32 + lane, tok0 = tok_tile(tile) * NT;
            const uint32_t src = tmem + d * NT + ((uint32_t)(quarter * 32) << 16);
            const int g0 = row - lane;                       // the warp's 32 rows
            const bool whole = g0 + 32 <= a.N && (g0 + 32 <= a.split || g0 >= a.split);
            const bool to32 = g0 >= a.split || a.y_f32;
            const bool packed = whole && !to32 && a.epi == kEpiNone && a.ldy % 2 == 0 && (reinterpret_cast<uintptr_t>(a.y) & 3) == 0;
#pragma unroll 1
            for (int c0 = half * HC; c0 < half * HC + HC && c0 < NT; c0 += CW) {
                if (!SPLIT && tok0 + c0 >= a.T) break;
                uint32_t v[CW / 16][16];
#pragma unroll
                for (int i = 0; i < CW / 16; ++i) tc::tmem_ld16(src + c0 + 16 * i, v[i]);
                tc::tmem_wait_ld();
                const int left = a.T - tok0 - c0;            // columns with a row of x
                if (SPLIT) {
#pragma unroll
                    for (int i = 0; i < CW; ++i) part[(c0 + i) * kTcRows + quarter * 32 + lane] = __uint_as_float(v[i / 16][i % 16]);
                } else if (a.epi == kEpiSwiglu) {
                    // even lanes hold gates, odd lanes the ups beside them: a pair of lanes exchanges one value each and
                    // finishes two columns
                    bf16* y = static_cast<bf16*>(a.y) + (long)(tok0 + c0 + (lane & 1)) * a.ldy + (row >> 1);
#pragma unroll
                    for (int i = 0; i < CW; i += 2) {
                        const float x0 = __uint_as_float(v[i / 16][i % 16]), x1 = __uint_as_float(v[i / 16][i % 16 + 1]);
                        const float got = __shfl_xor_sync(0xffffffffu, (lane & 1) ? x0 : x1, 1);
                        const float gate = (lane & 1) ? got : x0, up = (lane & 1) ? x1 : got;
                        if (row < a.N && i + (lane & 1) < left)
                            y[(long)i * a.ldy] = __float2bfloat16_rn(__fdividef(gate, 1.0f + __expf(-gate)) * up);
                    }
                } else if (packed) {   // two rows of one column per lane
                    bf16* y = static_cast<bf16*>(a.y) + (long)(tok0 + c0 + (lane & 1)) * a.ldy + (row & ~1);
#pragma unroll
                    for (int i = 0; i < CW; i += 2) {
                        const float x0 = __uint_as_float(v[i / 16][i % 16]), x1 = __uint_as_float(v[i / 16][i % 16 + 1]);
                        const float got = __shfl_xor_sync(0xffffffffu, (lane & 1) ? x0 : x1, 1);
                        if (i + (lane & 1) < left)
                            *reinterpret_cast<uint32_t*>(y + (long)i * a.ldy) = (lane & 1) ? pack_bf16(got, x1) : pack_bf16(x0, got);
                    }
                } else if (whole && to32 && a.epi == kEpiNone) {
                    const bool second = g0 >= a.split;
                    const long ld = second ? a.ldy32 : a.ldy;
                    float* y = (second ? a.y32 - a.split : static_cast<float*>(a.y)) + (long)(tok0 + c0) * ld + row;
#pragma unroll
                    for (int i = 0; i < CW; ++i)
                        if (i < left) y[(long)i * ld] = __uint_as_float(v[i / 16][i % 16]);
                } else if (row < a.N) {
#pragma unroll
                    for (int i = 0; i < CW; ++i)
                        if (i < left) store_out<false>(a, tok0 + c0 + i, row, __uint_as_float(v[i / 16][i % 16]));
                }
            }
            tc::tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(dempty(d));
        }
    }
    if (SPLIT) {
        cluster_sync_all();   // every CTA's partial tile is in its shared memory
        if (!*abort_flag) {
            pdl_wait();
            const int row0 = row_tile(first) * kTcRows, tok0 = tok_tile(first) * NT;
            const int c0 = NT * kpart / ksplit, c1 = NT * (kpart + 1) / ksplit;
            const uint32_t base = smem_u32(part);
            for (int i = c0 * kTcRows + t; i < c1 * kTcRows; i += kTcThreads) {
                float v = 0.f;
                for (int r = 0; r < ksplit; ++r) v += ld_dsmem(base + i * 4, r);
                const int tok = tok0 + i / kTcRows, row = row0 + i % kTcRows;
                if (a.epi == kEpiSwiglu) {   // 128 rows per column: neighbours in a warp are neighbouring rows
                    const float up = __shfl_down_sync(0xffffffffu, v, 1);
                    if (!(lane & 1) && row < a.N && tok < a.T)
                        static_cast<bf16*>(a.y)[(long)tok * a.ldy + (row >> 1)] = __float2bfloat16_rn(silu_f(v) * up);
                } else if (row < a.N && tok < a.T) {
                    store_out<false>(a, tok, row, v);
                }
            }
        }
        cluster_sync_all();   // nobody leaves while its tile may still be read
    }
    tc::tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc::tc_fence_after();
        tc::tmem_dealloc(tmem, COLS);
    }
    if (t == 0 && *abort_flag && status) *status = kStatusMbarTimeout;
}

}  // namespace lm
}  // namespace bw
