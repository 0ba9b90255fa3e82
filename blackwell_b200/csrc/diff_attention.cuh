// Differential attention: per query head two causal softmax maps over the last `window` positions, both over the same values,
//   o = a1 - lambda a2,   out = o / rms(o) * out_scale.
// A cached position is, per key / value head, [map 1 key | map 2 key | value], keys after rotation; position p sits in row
// p % cap of the slot's ring.
//   diff_prep_kernel     portions and 32-bit mode: rotates the queries in place, writes the new cache rows.
//   diff_decode_kernel   one token per sequence (bf16): rotation, cache row, attention and combination in one launch.  An MMA
//                        row tile is eight heads of one key / value head, map 1 in rows 0-7 and map 2 in rows 8-15, so that
//                        both maps of a head meet in the registers of one thread; each warp streams its own 16-key tiles
//                        by TMA, the context is split over a cluster whose blocks merge through distributed shared memory.
//   diff_flash_kernel    portions (bf16): flash attention with one half of the warps per map, combined through shared memory.
//   diff_scalar_kernel   32-bit mode and sizes the others do not take.
// Scores, softmax and sums are fp32; the softmax weights enter the MMA as a bf16 high part plus a bf16 remainder.
#pragma once
#include <cuda.h>

#include "gemm_w4a8_tc.cuh"
#include "lm_device.cuh"
#include "lm_ops.h"

namespace bw {
namespace lm {

// Element d of a head's rotated vector x: pairs (i, i + half) below rot, the rest passes.
template <typename A>
__device__ __forceinline__ float rot_half_elem(const A* x, int d, int rot, const float2* cs) {
    const float self = to_f(x[d]);
    if (d >= rot) return self;
    const int half = rot / 2;
    const float2 w = cs[d < half ? d : d - half];
    return d < half ? self * w.x - to_f(x[d + half]) * w.y : self * w.x + to_f(x[d - half]) * w.y;
}

// First visible position.
__device__ __forceinline__ int first_key(const DiffAttnArgs& a, int pos) { return a.window > 0 ? max(0, pos - a.window + 1) : 0; }

template <typename A, int VW>
__device__ __forceinline__ void load_vec(const A* p, float (&v)[VW]) {
    if constexpr (VW == 1) {
        v[0] = to_f(p[0]);
    } else {
        static_assert(VW == 8 && sizeof(A) == 2, "");
        const uint4 u = *reinterpret_cast<const uint4*>(p);
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            v[2 * i] = __uint_as_float(w[i] << 16);
            v[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
        }
    }
}
template <typename A, int VW>
__device__ __forceinline__ void store_vec(A* p, const float (&v)[VW]) {
    if constexpr (VW == 1) {
        p[0] = from_f<A>(v[0]);
    } else {
        *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
    }
}

// VW elements per thread: query pairs, key pairs, unrotated key elements, values.
template <typename A, int VW>
__global__ void __launch_bounds__(256) diff_prep_kernel(const DiffAttnArgs a, const Rows r) {
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.y, slot = r.slot_of(row), pos = r.pos_of(row);
    if (slot < 0 || pos >= a.max_seq) return;
    const int D8 = pad8(a.dim), V8 = pad8(a.V), half = a.rot_dims / 2, per = half / VW, rest = (D8 - a.rot_dims) / VW;
    const int nq = a.heads * 2 * per, nk = a.k ? a.kv_heads * 2 * per : 0, nr = a.k ? a.kv_heads * 2 * rest : 0;
    int i = blockIdx.x * 256 + threadIdx.x;
    const float2* cs = a.cs + (long)pos * half;
    A* entry = static_cast<A*>(a.cache) + ((long)slot * a.cap + pos % a.cap) * a.kv_heads * diff_row(a.dim, a.V);
    auto key_at = [&](int vec) { return entry + (vec >> 1) * diff_row(a.dim, a.V) + (vec & 1) * D8; };   // vec: head and map
    float u[VW], v[VW];
    if (i < nq + nk) {
        const bool isq = i < nq;
        if (!isq) i -= nq;
        const int vec = i / per, d = (i - vec * per) * VW;
        const A* src = (isq ? static_cast<const A*>(a.q) : static_cast<const A*>(a.k)) + (long)row * a.ld + vec * D8 + d;
        load_vec<A, VW>(src, u);
        load_vec<A, VW>(src + half, v);
#pragma unroll
        for (int e = 0; e < VW; ++e) {
            const float2 w = cs[d + e];
            const float x = u[e], y = v[e];
            u[e] = x * w.x - y * w.y;
            v[e] = y * w.x + x * w.y;
        }
        A* dst = isq ? static_cast<A*>(a.q) + (long)row * a.ld + vec * D8 + d : key_at(vec) + d;
        store_vec<A, VW>(dst, u);
        store_vec<A, VW>(dst + half, v);
    } else if (i < nq + nk + nr) {
        i -= nq + nk;
        const int vec = i / rest, d = a.rot_dims + (i - vec * rest) * VW;
        load_vec<A, VW>(static_cast<const A*>(a.k) + (long)row * a.ld + vec * D8 + d, u);
        store_vec<A, VW>(key_at(vec) + d, u);
    } else {
        i = (i - nq - nk - nr) * VW;
        if (!a.k || i >= a.kv_heads * V8) return;
        load_vec<A, VW>(static_cast<const A*>(a.v) + (long)row * a.ld + i, u);
        store_vec<A, VW>(key_at(2 * (i / V8)) + 2 * D8 + i % V8, u);
    }
}

// ------------------------------------------------------------------------------------------ any size, fp32 FMAs
constexpr int kDiffKeys = 32;
constexpr int kDiffCols = 8;   // value columns per thread: 2048 at most

// Block (head, row); rows prepared by diff_prep_kernel.
template <typename A>
__global__ void __launch_bounds__(256) diff_scalar_kernel(const DiffAttnArgs a, const Rows r) {
    extern __shared__ float sm[];
    const int D8 = pad8(a.dim), V8 = pad8(a.V), seg = diff_row(a.dim, a.V);
    float* q = sm;                      // [2][D8]
    float* sc = q + 2 * D8;             // [2][kDiffKeys]
    float* buf = sc + 2 * kDiffKeys;    // [32]
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31, h = blockIdx.x, row = blockIdx.y;
    pdl_trigger();
    pdl_wait();
    const int slot = r.slot_of(row), pos = min(r.pos_of(row), a.max_seq - 1);
    if (slot < 0) return;
    const A* cache = static_cast<const A*>(a.cache) + (long)slot * a.cap * a.kv_heads * seg + h / (a.heads / a.kv_heads) * seg;
    const long ldc = (long)a.kv_heads * seg;
    for (int i = t; i < 2 * D8; i += 256) q[i] = to_f(static_cast<const A*>(a.q)[(long)row * a.ld + h * 2 * D8 + i]);
    const int k0 = first_key(a, pos), r0 = k0 % a.cap;
    auto entry = [&](int key) {
        const int i = r0 + key - k0;
        return cache + (long)(i >= a.cap ? i - a.cap : i) * ldc;
    };
    float acc[2][kDiffCols] = {}, m[2] = {-INFINITY, -INFINITY}, l[2] = {};
    for (int kt = k0; kt <= pos; kt += kDiffKeys) {
        const int n = min(kDiffKeys, pos + 1 - kt);
        __syncthreads();
        for (int j = warp; j < 2 * n; j += 8) {
            const A* e = entry(kt + (j >> 1)) + (j & 1) * D8;
            const float* qm = q + (j & 1) * D8;
            float s = 0.f;
            for (int i = lane; i < D8; i += 32) s = fmaf(qm[i], to_f(e[i]), s);
            s = warp_sum(s);
            if (lane == 0) sc[(j & 1) * kDiffKeys + (j >> 1)] = s * a.scale;
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            float mn = m[i];
            for (int j = 0; j < n; ++j) mn = fmaxf(mn, sc[i * kDiffKeys + j]);
            const float alpha = expf(m[i] - mn);
            m[i] = mn;
            l[i] *= alpha;
#pragma unroll
            for (int c = 0; c < kDiffCols; ++c) acc[i][c] *= alpha;
        }
        for (int j = 0; j < n; ++j) {
            const float p0 = expf(sc[j] - m[0]), p1 = expf(sc[kDiffKeys + j] - m[1]);
            l[0] += p0;
            l[1] += p1;
            const A* v = entry(kt + j) + 2 * D8;
#pragma unroll
            for (int c = 0; c < kDiffCols; ++c)
                if (c * 256 + t < V8) {
                    const float x = to_f(v[c * 256 + t]);
                    acc[0][c] = fmaf(p0, x, acc[0][c]);
                    acc[1][c] = fmaf(p1, x, acc[1][c]);
                }
        }
    }
    float ss = 0.f;
    const float f0 = 1.0f / l[0], f1 = a.lambda / l[1];
#pragma unroll
    for (int c = 0; c < kDiffCols; ++c) {
        acc[0][c] = acc[0][c] * f0 - acc[1][c] * f1;
        ss = fmaf(acc[0][c], acc[0][c], ss);
    }
    const float f = a.out_scale / sqrtf(block_sum(ss, buf) / (float)a.V + a.eps);
    A* out = static_cast<A*>(a.out) + (long)row * a.ldout + h * V8;
#pragma unroll
    for (int c = 0; c < kDiffCols; ++c)
        if (c * 256 + t < V8) out[c * 256 + t] = from_f<A>(acc[0][c] * f);
}

// ------------------------------------------------------------------------------------------ decode
constexpr int kDiffTile = 16;    // positions per tile of a warp, from a multiple of 16 on
struct DiffDecodeSmem {          // queries, new cache entry, stats, barriers, then the warps' tiles (later their partial outputs)
    int qrow, boxes, tile, new_off, st_off, bar_off, ring_off, total;   // a tile: boxes of 16 rows x 64 columns, swizzled
    __host__ __device__ DiffDecodeSmem(int dim, int V, int VT, int warps, int stages) {
        boxes = (diff_row(dim, V) + 63) / 64;
        tile = boxes * kDiffTile * 128;
        qrow = pad16(dim) * 2 + 16;
        new_off = 16 * qrow;
        st_off = new_off + boxes * 128;                // [warps][16] maximum, sum; [warps][16] weights; the block's [16] maximum, sum
        bar_off = st_off + warps * 16 * 12 + 16 * 8;
        ring_off = (bar_off + warps * stages * 8 + 1023) & ~1023;
        const int ring = warps * stages * tile + 2048, part = warps * 16 * VT * 8 * 4;   // a value fragment may start one box past the tile
        total = 1024 + ring_off + (ring > part ? ring : part);   // 1024: alignment of the base
    }
};

// Block (split, key / value head and eight of its query heads, row); WARPS warps, each with tiles and softmax state of its own.
// KS: 16-wide query steps per map; VT: value columns / 8.
template <int KS, int VT, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) diff_decode_kernel(const __grid_constant__ CUtensorMap map, const DiffAttnArgs a, const Rows r,
                                                                 int stages, int* status) {
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    const DiffDecodeSmem L(a.dim, a.V, VT, WARPS, stages);
    const int D8 = pad8(a.dim), D16 = pad16(a.dim), V8 = pad8(a.V), seg = diff_row(a.dim, a.V), group = a.heads / a.kv_heads;
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, q4 = lane & 3;
    const int htiles = (group + 7) / 8, kvh = blockIdx.y / htiles, h0 = (blockIdx.y - kvh * htiles) * 8, nh = min(8, group - h0);
    const int split = blockIdx.x, row = blockIdx.z, half = a.rot_dims / 2;
    const uint32_t sb = smem_u32(smem), bars = sb + L.bar_off + warp * stages * 8, ring = sb + L.ring_off + warp * stages * L.tile;
    float2* stats = reinterpret_cast<float2*>(smem + L.st_off);
    float* weights = reinterpret_cast<float*>(stats + WARPS * 16);
    float2* block_stats = reinterpret_cast<float2*>(weights + WARPS * 16);
    if (lane == 0) {
        for (int i = 0; i < stages; ++i) mbar_init(bars + 8 * i, 1);
        mbar_fence_init();
    }
    __syncwarp();
    pdl_trigger();
    pdl_wait();
    const int slot = r.slot_of(row), pos = min(r.pos_of(row), a.max_seq - 1);
    if (slot < 0) return;                                         // the whole cluster
    const int k0 = first_key(a, pos), tile0 = k0 / kDiffTile, tiles = pos / kDiffTile - tile0 + 1, per = (tiles + a.splits - 1) / a.splits;
    const int t0 = tile0 + split * per, t1 = min(tile0 + tiles, t0 + per);
    const int fresh = a.k ? pos - 1 : pos;                        // last position that comes from the cache
    int waited = 0, issued = 0;
    auto issue = [&](int tile) {   // lane 0
        const int s = issued % stages, y = slot * a.cap + (int)((long)tile * kDiffTile % a.cap);
        mbar_expect_tx(bars + 8 * s, L.tile);
        for (int b = 0; b < L.boxes; ++b) tc::tma_load_2d(ring + s * L.tile + b * kDiffTile * 128, &map, kvh * seg + b * 64, y, bars + 8 * s);
    };
    int next = t0 + warp;
    for (; issued < stages && next < t1; next += WARPS, ++issued)
        if (lane == 0) issue(next);
    // rotated queries: row = map * 8 + head
    const float2* cs = a.cs + (long)pos * half;
#pragma unroll 4
    for (int i = t; i < 16 * D16; i += WARPS * 32) {
        const int qr = i / D16, d = i - qr * D16, hh = qr & 7;
        float v = 0.f;
        if (hh < nh && d < D8) {
            const bf16* q = static_cast<const bf16*>(a.q) + (long)row * a.ld + (2L * (kvh * group + h0 + hh) + (qr >> 3)) * D8;
            v = rot_half_elem(q, d, a.rot_dims, cs);
        }
        *reinterpret_cast<bf16*>(smem + qr * L.qrow + d * 2) = __float2bfloat16_rn(v);
    }
    if (a.k && t1 == tile0 + tiles && t0 < t1) {   // the newest position's entry
        const bf16* k = static_cast<const bf16*>(a.k) + (long)row * a.ld + 2L * kvh * D8;
        const bf16* v = static_cast<const bf16*>(a.v) + (long)row * a.ld + kvh * V8;
        bf16* entry = static_cast<bf16*>(a.cache) + (((long)slot * a.cap + pos % a.cap) * a.kv_heads + kvh) * seg;
        for (int i = t; i < L.boxes * 64; i += WARPS * 32) {
            bf16 x = __float2bfloat16_rn(0.f);
            if (i < 2 * D8) x = __float2bfloat16_rn(rot_half_elem(k + (i < D8 ? 0 : D8), i < D8 ? i : i - D8, a.rot_dims, cs));
            else if (i < seg) x = v[i - 2 * D8];
            *reinterpret_cast<bf16*>(smem + L.new_off + i * 2) = x;
            if (h0 == 0 && i < seg) entry[i] = x;
        }
    }
    __syncthreads();
    uint32_t qa[KS][2], qb[KS][2];         // map 1: rows 0-7 of the MMA tile, map 2: rows 8-15
#pragma unroll
    for (int i = 0; i < KS; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int off = g * L.qrow + (i * 16 + e * 8 + 2 * q4) * 2;
            qa[i][e] = i * 16 < D16 ? *reinterpret_cast<const uint32_t*>(smem + off) : 0u;
            qb[i][e] = i * 16 < D16 ? *reinterpret_cast<const uint32_t*>(smem + 8 * L.qrow + off) : 0u;
        }
    float O[VT][4] = {};
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {};
    const float sl2 = a.scale * 1.4426950408889634f;   // softmax in base 2
    CopyWait copied{status};
    const int krow = (lane & 7) + (lane >> 4) * 8, kc = (lane >> 3) & 1, vrow = lane & 15, vc = lane >> 4;
    for (int tile = t0 + warp; tile < t1; tile += WARPS) {
        const int s_ = waited % stages, j0 = tile * kDiffTile;
        const uint32_t kb = ring + s_ * L.tile;
        copied(bars + 8 * s_, (waited / stages) & 1);
        ++waited;
        if (j0 < k0 || j0 + kDiffTile - 1 > fresh) {   // rows that are not visible become zeros, the newest one its entry
            unsigned char* dst = smem + (kb - sb);
            for (int i = lane; i < L.boxes * kDiffTile * 8; i += 32) {
                const int c = i & 7, rr = (i >> 3) & 15, b = i >> 7, p = j0 + rr;
                if (p < k0 || p > fresh)
                    *reinterpret_cast<uint4*>(dst + b * kDiffTile * 128 + rr * 128 + ((c ^ (rr & 7)) << 4)) =
                        p == pos ? *reinterpret_cast<const uint4*>(smem + L.new_off + b * 128 + c * 16) : make_uint4(0, 0, 0, 0);
            }
            fence_proxy_async();   // before the next copy into this buffer
            __syncwarp();
        }
        // 16-byte column chunk `chunk` of tile row `rr`
        auto at = [&](int rr, int chunk) { return kb + (chunk >> 3) * (kDiffTile * 128) + rr * 128 + (((chunk ^ rr) & 7) << 4); };
        float s[4][4] = {};            // two accumulators per eight keys: one per map
#pragma unroll
        for (int i = 0; i < KS; ++i)
            if (i * 16 < D16) {
                uint32_t b[4], c[4];
                ldsm4(at(krow, 2 * i + kc), b);
                ldsm4(at(krow, D8 / 8 + 2 * i + kc), c);
                mma_bf16(s[0], qa[i][0], 0u, qa[i][1], 0u, b[0], b[1]);
                mma_bf16(s[1], qa[i][0], 0u, qa[i][1], 0u, b[2], b[3]);
                mma_bf16(s[2], 0u, qb[i][0], 0u, qb[i][1], c[0], c[1]);
                mma_bf16(s[3], 0u, qb[i][0], 0u, qb[i][1], c[2], c[3]);
            }
        float alpha[2];
#pragma unroll
        for (int p = 0; p < 2; ++p) {
            float mx = m[p], x[4];
#pragma unroll
            for (int c = 0; c < 2; ++c)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int key = j0 + 8 * c + 2 * q4 + e;
                    x[2 * c + e] = key >= k0 && key <= pos ? s[2 * p + c][2 * p + e] * sl2 : -INFINITY;
                    mx = fmaxf(mx, x[2 * c + e]);
                }
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));   // finite: every tile holds a visible position
            alpha[p] = exp2_fast(m[p] - mx);
            m[p] = mx;
            float sum = 0.f;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                x[e] = exp2_fast(x[e] - mx);
                sum += x[e];
            }
            l[p] = l[p] * alpha[p] + sum;
            s[0][2 * p] = x[0];
            s[0][2 * p + 1] = x[1];
            s[1][2 * p] = x[2];
            s[1][2 * p + 1] = x[3];
        }
        if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
            for (int j = 0; j < VT; ++j) { O[j][0] *= alpha[0]; O[j][1] *= alpha[0]; O[j][2] *= alpha[1]; O[j][3] *= alpha[1]; }
        }
        uint32_t ph[4], pl[4];
        split_bf16(s[0][0], s[0][1], ph[0], pl[0]);
        split_bf16(s[0][2], s[0][3], ph[1], pl[1]);
        split_bf16(s[1][0], s[1][1], ph[2], pl[2]);
        split_bf16(s[1][2], s[1][3], ph[3], pl[3]);
#pragma unroll
        for (int j = 0; j < VT; j += 2)
            if (8 * j < V8) {
                uint32_t v[4];
                ldsm4t(at(vrow, D8 / 4 + j + vc), v);
                mma_bf16(O[j], ph[0], ph[1], ph[2], ph[3], v[0], v[1]);
                mma_bf16(O[j + 1], ph[0], ph[1], ph[2], ph[3], v[2], v[3]);
                mma_bf16(O[j], pl[0], pl[1], pl[2], pl[3], v[0], v[1]);
                mma_bf16(O[j + 1], pl[0], pl[1], pl[2], pl[3], v[2], v[3]);
            }
        __syncwarp();                  // everybody is done with the buffer
        if (next < t1) {
            if (lane == 0) issue(next);
            ++issued;
            next += WARPS;
        }
    }
    if (copied.dead)                   // gave up: copies still in flight land before the buffers are used for something else
        for (; waited < issued; ++waited) mbar_wait(bars + 8 * (waited % stages), (waited / stages) & 1);
    // merge: the warps of the block, then the blocks of the cluster
#pragma unroll
    for (int p = 0; p < 2; ++p) {
        l[p] += __shfl_xor_sync(0xffffffffu, l[p], 1);
        l[p] += __shfl_xor_sync(0xffffffffu, l[p], 2);
        if (q4 == 0) stats[warp * 16 + g + 8 * p] = make_float2(m[p], l[p]);
    }
    __syncthreads();   // everybody is done with the tiles
    constexpr int kRow = VT * 8;
    float* part = reinterpret_cast<float*>(smem + L.ring_off);   // [warp][16][kRow]
#pragma unroll
    for (int j = 0; j < VT; ++j) {
        float* o = part + (warp * 16 + g) * kRow + 8 * j + 2 * q4;
        *reinterpret_cast<float2*>(o) = make_float2(O[j][0], O[j][1]);
        *reinterpret_cast<float2*>(o + 8 * kRow) = make_float2(O[j][2], O[j][3]);
    }
    if (t < 16) {
        float mx = -INFINITY, sum = 0.f;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) mx = fmaxf(mx, stats[w * 16 + t].x);
#pragma unroll
        for (int w = 0; w < WARPS; ++w) {
            const float2 st = stats[w * 16 + t];
            const float f = st.y > 0.f ? exp2_fast(st.x - mx) : 0.f;   // a warp without tiles has neither
            weights[w * 16 + t] = f;
            sum = fmaf(f, st.y, sum);
        }
        block_stats[t] = make_float2(mx, sum);
    }
    __syncthreads();
    for (int rr = warp; rr < 16; rr += WARPS) {
        if ((rr & 7) >= nh) continue;
        for (int c = lane * 4; c < V8; c += 128) {   // these four columns are read and written by this thread alone
            float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int w = 0; w < WARPS; ++w) {
                const float f = weights[w * 16 + rr];
                const float4 x = *reinterpret_cast<const float4*>(part + (w * 16 + rr) * kRow + c);
                o.x = fmaf(f, x.x, o.x);
                o.y = fmaf(f, x.y, o.y);
                o.z = fmaf(f, x.z, o.z);
                o.w = fmaf(f, x.w, o.w);
            }
            *reinterpret_cast<float4*>(part + rr * kRow + c) = o;
        }
    }
    cluster_sync_all();
    constexpr int kCols = (VT + 3) / 4;
    const uint32_t st = smem_u32(block_stats), pb = sb + L.ring_off;
    for (int hh = split + a.splits * warp; hh < nh; hh += a.splits * WARPS) {
        // lane = 4 * block + 2 * map + (maximum, sum)
        const int src = lane >> 2, p = (lane >> 1) & 1;
        const float v = src < a.splits ? ld_dsmem(st + (hh + 8 * p) * 8 + (lane & 1) * 4, src) : 0.f;
        const float lm = __shfl_sync(0xffffffffu, v, lane & ~1), ls = __shfl_sync(0xffffffffu, v, lane | 1);
        float mx = ls > 0.f ? lm : -INFINITY;   // a block without tiles has neither
#pragma unroll
        for (int o = 4; o < 32; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        float f = ls > 0.f ? exp2_fast(lm - mx) : 0.f, sum = f * ls;
#pragma unroll
        for (int o = 4; o < 32; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        f *= (p ? -a.lambda : 1.0f) / sum;
        float o[kCols] = {}, ss = 0.f;
        for (int s = 0; s < a.splits; ++s) {
            const float f0 = __shfl_sync(0xffffffffu, f, 4 * s), f1 = __shfl_sync(0xffffffffu, f, 4 * s + 2);
            if (f0 == 0.f && f1 == 0.f) continue;
            float x[2][kCols];
#pragma unroll
            for (int j = 0; j < kCols; ++j) {
                const int c = min(32 * j + lane, V8 - 1);
                x[0][j] = ld_dsmem(pb + (hh * kRow + c) * 4, s);
                x[1][j] = ld_dsmem(pb + ((hh + 8) * kRow + c) * 4, s);
            }
#pragma unroll
            for (int j = 0; j < kCols; ++j) o[j] = fmaf(f0, x[0][j], fmaf(f1, x[1][j], o[j]));
        }
#pragma unroll
        for (int j = 0; j < kCols; ++j)
            if (32 * j + lane < V8) ss = fmaf(o[j], o[j], ss);
        const float scale = a.out_scale / sqrtf(warp_sum(ss) / (float)a.V + a.eps);
        bf16* out = static_cast<bf16*>(a.out) + (long)row * a.ldout + (kvh * group + h0 + hh) * V8;
#pragma unroll
        for (int j = 0; j < kCols; ++j)
            if (32 * j + lane < V8) out[32 * j + lane] = __float2bfloat16_rn(o[j] * scale);
    }
    cluster_sync_all();   // nobody leaves while its partial result may still be read
}

// ------------------------------------------------------------------------------------------ portions
struct DiffFlashSmem {
    int row, vrow, k_off, kbuf, xrow, total;
    __host__ __device__ DiffFlashSmem(int dim, int VT, int MT, int KK) {
        row = 2 * pad16(dim) * 2 + 16;
        vrow = VT * 16 + 16;
        k_off = 64 * MT * row;
        kbuf = KK * (row + vrow);
        xrow = VT * 8 + 4;                       // floats of a row of the second map's output
        total = k_off + 2 * kbuf;
        if (total < 64 * MT * xrow * 4) total = 64 * MT * xrow * 4;
    }
};

// Block (head, 64 * MT query rows); a warp has MT tiles of 16 rows of one map (warps 0-3 map 1, warps 4-7 map 2), so that every
// key and value fragment it reads from shared memory serves MT products.  KK: keys per shared-memory tile.
template <int VT, int MT, int KK>
__global__ void __launch_bounds__(256, 1) diff_flash_kernel(const DiffAttnArgs a, const Rows r) {
    extern __shared__ __align__(16) unsigned char smem[];
    constexpr int kQ = 64 * MT, KT = 4;   // KT: 8-key tiles per softmax step
    const int D8 = pad8(a.dim), D16 = pad16(a.dim), V8 = pad8(a.V), seg = diff_row(a.dim, a.V);
    const DiffFlashSmem L(a.dim, VT, MT, KK);
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, q4 = lane & 3, map = warp >> 2;
    const int q0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * kQ, h = blockIdx.x;   // longest rows first
    const uint32_t sb = smem_u32(smem);
    const long ldc = (long)a.kv_heads * seg;
    const bf16* cache = static_cast<const bf16*>(a.cache) + (long)r.slot * a.cap * ldc + h / (a.heads / a.kv_heads) * seg;
    const int last = min(r.T, q0 + kQ) - 1;                  // last real query row of the block
    const int kmin = first_key(a, r.pos0 + q0), kend = r.pos0 + last + 1, ring0 = kmin % a.cap;
    const int tiles = (kend - kmin + KK - 1) / KK;
    pdl_trigger();
    pdl_wait();
    const RowWalk qwalk(t, 256, D16 / 4), vwalk(t, 256, VT);
    auto entry = [&](int key) {
        int i = ring0 + key - kmin;
        if (i >= a.cap) i -= a.cap;
        return cache + i * ldc;
    };
    auto issue = [&](int tile, int buf) {
        const uint32_t kb = sb + L.k_off + buf * L.kbuf, vb = kb + KK * L.row;
        for (RowWalk w = qwalk; w.row < KK; w.next()) {      // both maps' keys, each padded to D16 columns
            const int c = w.col * 8, cm = c < D16 ? c : c - D16, key = kmin + tile * KK + w.row;
            const bool ok = key < kend && cm < D8;
            cp_async16z(kb + w.row * L.row + c * 2, ok ? entry(key) + (c < D16 ? 0 : D8) + cm : cache, ok);
        }
        for (RowWalk w = vwalk; w.row < KK; w.next()) {
            const int c = w.col * 8, key = kmin + tile * KK + w.row;
            const bool ok = key < kend && c < V8;
            cp_async16z(vb + w.row * L.vrow + c * 2, ok ? entry(key) + 2 * D8 + c : cache, ok);
        }
        cp_async_commit();
    };
    for (RowWalk w = qwalk; w.row < kQ; w.next()) {
        const int c = w.col * 8, cm = c < D16 ? c : c - D16;
        const bool ok = q0 + w.row < r.T && cm < D8;
        const bf16* src = static_cast<const bf16*>(a.q);
        cp_async16z(sb + w.row * L.row + c * 2, ok ? src + (long)(q0 + w.row) * a.ld + (2 * h + (c < D16 ? 0 : 1)) * D8 + cm : src, ok);
    }
    issue(0, 0);
    float O[MT][VT][4] = {};
    float m[MT][2], l[MT][2];
#pragma unroll
    for (int i = 0; i < MT; ++i) { m[i][0] = m[i][1] = -INFINITY; l[i][0] = l[i][1] = 0.f; }
    const int wr = 16 * MT * (warp & 3), wpos = r.pos0 + q0 + wr;   // the warp's first query row and its position
    const int window = a.window > 0 ? a.window : 0x7fffffff;
    const float sl2 = a.scale * 1.4426950408889634f;                // softmax in base 2
    for (int tile = 0; tile < tiles; ++tile) {
        const int buf = tile & 1;
        const uint32_t kb = sb + L.k_off + buf * L.kbuf, vb = kb + KK * L.row;
        cp_async_wait<0>();
        __syncthreads();
        if (tile + 1 < tiles) issue(tile + 1, buf ^ 1);
#pragma unroll 1
        for (int sub = 0; sub < KK; sub += 8 * KT) {
            const int key0 = kmin + tile * KK + sub;
            if (key0 > wpos + 16 * MT - 1) break;            // nothing more of this tile is visible to the warp
            if (wpos - (key0 + 8 * KT - 1) >= window) continue;   // all of it has left the window of every row
            float s[MT][KT][4] = {};
#pragma unroll 2
            for (int k0 = 0; k0 < D16; k0 += 16) {
                uint32_t fa[MT][4];
#pragma unroll
                for (int i = 0; i < MT; ++i)
                    ldsm4(sb + (wr + 16 * i + (lane & 15)) * L.row + (map * D16 + k0 + (lane >> 4) * 8) * 2, fa[i]);
#pragma unroll
                for (int jj = 0; jj < KT / 2; ++jj) {
                    uint32_t fb[4];
                    ldsm4(kb + (sub + 16 * jj + (lane & 7) + (lane >> 4) * 8) * L.row + (map * D16 + k0 + ((lane >> 3) & 1) * 8) * 2, fb);
#pragma unroll
                    for (int i = 0; i < MT; ++i) {
                        mma_bf16(s[i][2 * jj], fa[i][0], fa[i][1], fa[i][2], fa[i][3], fb[0], fb[1]);
                        mma_bf16(s[i][2 * jj + 1], fa[i][0], fa[i][1], fa[i][2], fa[i][3], fb[2], fb[3]);
                    }
                }
            }
            const bool edge = key0 + 8 * KT - 1 > wpos || wpos + 16 * MT - 1 - key0 >= window;
#pragma unroll
            for (int i = 0; i < MT; ++i)
#pragma unroll
                for (int p = 0; p < 2; ++p) {
                    const int pos = wpos + 16 * i + g + 8 * p;
                    float mx = m[i][p];
#pragma unroll
                    for (int j = 0; j < KT; ++j)
#pragma unroll
                        for (int e = 0; e < 2; ++e) {
                            float& x = s[i][j][2 * p + e];
                            const int key = key0 + 8 * j + 2 * q4 + e;
                            x *= sl2;
                            if (edge && (key > pos || pos - key >= window)) x = -INFINITY;
                            mx = fmaxf(mx, x);
                        }
                    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                    const float base = mx == -INFINITY ? 0.f : mx, alpha = exp2_fast(m[i][p] - base);
                    m[i][p] = mx;
                    float sum = 0.f;
#pragma unroll
                    for (int j = 0; j < KT; ++j)
#pragma unroll
                        for (int e = 0; e < 2; ++e) {
                            float& x = s[i][j][2 * p + e];
                            x = exp2_fast(x - base);
                            sum += x;
                        }
                    l[i][p] = l[i][p] * alpha + sum;
                    if (__any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll
                        for (int j = 0; j < VT; ++j) { O[i][j][2 * p] *= alpha; O[i][j][2 * p + 1] *= alpha; }
                    }
                }
#pragma unroll
            for (int kk = 0; kk < KT / 2; ++kk) {   // 16 keys: the score fragments are the A operand
                uint32_t ph[MT][4], pl[MT][4];
#pragma unroll
                for (int i = 0; i < MT; ++i) {
                    split_bf16(s[i][2 * kk][0], s[i][2 * kk][1], ph[i][0], pl[i][0]);
                    split_bf16(s[i][2 * kk][2], s[i][2 * kk][3], ph[i][1], pl[i][1]);
                    split_bf16(s[i][2 * kk + 1][0], s[i][2 * kk + 1][1], ph[i][2], pl[i][2]);
                    split_bf16(s[i][2 * kk + 1][2], s[i][2 * kk + 1][3], ph[i][3], pl[i][3]);
                }
#pragma unroll
                for (int j = 0; j < VT; j += 2) {
                    uint32_t v[4];
                    ldsm4t(vb + (sub + 16 * kk + (lane & 15)) * L.vrow + (8 * j + (lane >> 4) * 8) * 2, v);
#pragma unroll
                    for (int i = 0; i < MT; ++i) {
                        mma_bf16(O[i][j], ph[i][0], ph[i][1], ph[i][2], ph[i][3], v[0], v[1]);
                        mma_bf16(O[i][j + 1], ph[i][0], ph[i][1], ph[i][2], ph[i][3], v[2], v[3]);
                        mma_bf16(O[i][j], pl[i][0], pl[i][1], pl[i][2], pl[i][3], v[0], v[1]);
                        mma_bf16(O[i][j + 1], pl[i][0], pl[i][1], pl[i][2], pl[i][3], v[2], v[3]);
                    }
                }
            }
        }
    }
    // o = a1 - lambda a2: the second map's warps hand their part over
    __syncthreads();
    float* x2 = reinterpret_cast<float*>(smem);
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int p = 0; p < 2; ++p) {
            float tot = l[i][p];
            tot += __shfl_xor_sync(0xffffffffu, tot, 1);
            tot += __shfl_xor_sync(0xffffffffu, tot, 2);
            l[i][p] = tot > 0.f ? (map ? a.lambda : 1.0f) / tot : 0.f;   // rows past the end may have seen nothing
            if (map) {
                float* d = x2 + (wr + 16 * i + g + 8 * p) * L.xrow + 2 * q4;
#pragma unroll
                for (int j = 0; j < VT; ++j) *reinterpret_cast<float2*>(d + 8 * j) = make_float2(O[i][j][2 * p] * l[i][p], O[i][j][2 * p + 1] * l[i][p]);
            }
        }
    __syncthreads();
    if (map) return;
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int p = 0; p < 2; ++p) {
            const int rr = wr + 16 * i + g + 8 * p, q = q0 + rr;
            const float* d = x2 + rr * L.xrow + 2 * q4;
            float ss = 0.f;
#pragma unroll
            for (int j = 0; j < VT; ++j) {
                const float2 b = *reinterpret_cast<const float2*>(d + 8 * j);
                O[i][j][2 * p] = O[i][j][2 * p] * l[i][p] - b.x;
                O[i][j][2 * p + 1] = O[i][j][2 * p + 1] * l[i][p] - b.y;
                ss = fmaf(O[i][j][2 * p], O[i][j][2 * p], fmaf(O[i][j][2 * p + 1], O[i][j][2 * p + 1], ss));
            }
            ss += __shfl_xor_sync(0xffffffffu, ss, 1);
            ss += __shfl_xor_sync(0xffffffffu, ss, 2);
            if (q >= r.T) continue;
            const float f = a.out_scale / sqrtf(ss / (float)a.V + a.eps);
            bf16* out = static_cast<bf16*>(a.out) + (long)q * a.ldout + h * V8;
#pragma unroll
            for (int j = 0; j < VT; ++j) {
                const int col = 8 * j + 2 * q4;
                if (col < V8) *reinterpret_cast<uint32_t*>(out + col) = pack_bf16(O[i][j][2 * p] * f, O[i][j][2 * p + 1] * f);
            }
        }
}

}  // namespace lm
}  // namespace bw
