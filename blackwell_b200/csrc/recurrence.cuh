// Gated linear recurrence  S_t = exp(a_t) S_(t-1) + w_t k_t v_t^T,  o_t = S_t^T q_t + D v_t  with an fp32 state per
// head, N x V.  Mamba-2 (a_t, w_t from the token, q / k shared by a group of heads) and retention (constant a per head)
// are both instances; the delta rule replaces w_t v_t by w_t (v_t - exp(a_t) S_(t-1)^T k_t), with unit vectors k and q.
//   recurrence_step_kernel   one token per sequence (decode) or a short / 32-bit run of tokens: the state tile of a CTA
//                            stays in registers, fp32 FMAs.  CONV: the convolution over the last inputs, silu and the
//                            step size are computed in the same launch.  DELTA: both products of the state (with k and with
//                            q) are taken before the write, o = S'^T q + (k q) u, so that one reduction serves both.
//   recurrence_chunk_kernel  prompts: 64 tokens at a time on the tensor cores (mma.sync bf16).  q, k and v are bf16 values;
//                            the decayed scores, the weighted values and the state enter their products as a bf16 high part
//                            plus a bf16 remainder.  State, decays and sums are fp32.
#pragma once
#include "lm_device.cuh"
#include "lm_ops.h"

namespace bw {
namespace lm {

constexpr int kRecV = 32;      // state columns per CTA
constexpr int kRecThreads = 256;

// NR: state rows per thread (rows n = ng + 32 i of 32 row groups); 8 lanes hold 4 columns each.
template <typename A, int NR, bool CONV, bool DELTA>
__global__ void __launch_bounds__(kRecThreads) recurrence_step_kernel(const RecurrenceArgs a, const ConvArgs c, const Rows r) {
    extern __shared__ float sm[];
    const int N = a.N, N8 = pad8(a.N), V8 = pad8(a.V);
    float* qs = sm;                 // [32 * NR] (zero beyond N)
    float* ks = qs + 32 * NR;
    float* vs = ks + 32 * NR;       // [32]
    float* red = vs + kRecV;        // [2][8 warps][32], DELTA: once for k, once for q
    constexpr int kRed = (DELTA ? 2 : 1) * 8 * kRecV;
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31;
    const int c4 = (lane & 7) * 4, ng = warp * 4 + (lane >> 3);
    const int h = blockIdx.y, v0 = blockIdx.x * kRecV;
    const int row0 = CONV || r.row_slot ? blockIdx.z : 0, nrows = CONV || r.row_slot ? 1 : r.T;
    const int grp = h / (a.heads / a.groups);
    const bool colv = v0 + c4 < V8;
    pdl_trigger();
    pdl_wait();
    const int slot = r.slot_of(row0), pos0 = r.pos_of(row0);
    if (slot < 0) return;
    float* Sg = a.S + (((long)slot * a.heads + h) * N) * V8 + v0 + c4;
    float4 S[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int n = ng + 32 * i;
        S[i] = pos0 > 0 && colv && n < N ? *reinterpret_cast<const float4*>(Sg + (long)n * V8) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float Dh = a.D ? a.D[h] : 0.f;
    for (int rr = 0; rr < nrows; ++rr) {
        const int row = row0 + rr;
        float la, w;
        if (CONV) {
            // channels this head needs: kRecV of v, N of k, N of q
            const int inner = c.heads * c.V, channels = inner + 2 * c.groups * N;
            const A* u = static_cast<const A*>(c.u) + (long)row * c.ldu + c.off;
            float* ring = c.ring + (long)slot * c.taps * channels;
            for (int i = t; i < kRecV + 64 * NR; i += kRecThreads) {
                int ch = -1, col = 0;
                bool keep = false;   // exactly one CTA stores a channel's input
                if (i < kRecV) {
                    if (v0 + i < a.V) { ch = h * a.V + v0 + i; col = h * V8 + v0 + i; keep = true; }
                } else {
                    const int part = (i - kRecV) / (32 * NR), n = (i - kRecV) - part * 32 * NR;
                    if (n < N) {
                        ch = inner + (part * c.groups + grp) * N + n;
                        col = c.heads * V8 + (part * c.groups + grp) * N8 + n;
                        keep = h % (a.heads / a.groups) == 0 && v0 == 0;
                    }
                }
                float y = 0.f;
                if (ch >= 0) {
                    const float now = to_f(u[col]);
                    y = c.bias ? c.bias[ch] : 0.f;
                    for (int j = 0; j < c.taps - 1; ++j) {
                        const int p = pos0 - (c.taps - 1) + j;
                        if (p >= 0) y = fmaf(c.w[ch * c.taps + j], ring[(long)(p % c.taps) * channels + ch], y);
                    }
                    y = fmaf(c.w[ch * c.taps + c.taps - 1], now, y);
                    y = to_f(from_f<A>(silu_f(y)));
                    if (keep) ring[(long)(pos0 % c.taps) * channels + ch] = now;   // an entry no other read of this step touches
                }
                if (i < kRecV) vs[i] = y;
                else if (i < kRecV + 32 * NR) ks[i - kRecV] = y;
                else qs[i - kRecV - 32 * NR] = y;
            }
            const float dt = softplus_f(c.dt_raw[(long)row * c.ld_dt + h] + c.dt_bias[h]);
            la = -expf(c.A_log[h]) * dt;
            w = c.beta_raw ? sigmoid_f(c.beta_raw[(long)row * c.ld_dt + h]) : dt;
        } else {
            const A* q = static_cast<const A*>(a.q) + (long)row * a.ldq + grp * N8;
            const A* k = static_cast<const A*>(a.k) + (long)row * a.ldk + grp * N8;
            const A* v = static_cast<const A*>(a.v) + (long)row * a.ldv + h * V8 + v0;
            for (int i = t; i < 32 * NR; i += kRecThreads) {
                qs[i] = i < N ? to_f(q[i]) : 0.f;
                ks[i] = i < N ? to_f(k[i]) : 0.f;
            }
            if (t < kRecV) vs[t] = v0 + t < a.V ? to_f(v[t]) : 0.f;
            la = a.log_decay ? a.log_decay[(long)row * a.heads + h] : a.head_log_decay[h];
            w = a.log_decay ? a.weight[(long)row * a.heads + h] : a.const_weight;
        }
        __syncthreads();
        const float d = expf(la);
        const float4 v = *reinterpret_cast<const float4*>(vs + c4);
        float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
        if (DELTA) {
            float sq = 0.f, sk = 0.f, kq = 0.f;
            for (int i = lane; i < 32 * NR; i += 32) {
                const float qi = qs[i], ki = ks[i];
                sq = fmaf(qi, qi, sq);
                sk = fmaf(ki, ki, sk);
                kq = fmaf(ki, qi, kq);
            }
            const float rq = a.q_scale / sqrtf(warp_sum(sq) + a.unit_eps), rk = 1.0f / sqrtf(warp_sum(sk) + a.unit_eps);
            kq = warp_sum(kq) * rq * rk;
            float kn[NR];
            float4 z = make_float4(0.f, 0.f, 0.f, 0.f);   // S'^T k, y: S'^T q
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                const int n = ng + 32 * i;
                const float qn = qs[n] * rq;
                kn[i] = ks[n] * rk;
                S[i].x *= d;
                S[i].y *= d;
                S[i].z *= d;
                S[i].w *= d;
                z.x = fmaf(S[i].x, kn[i], z.x);
                z.y = fmaf(S[i].y, kn[i], z.y);
                z.z = fmaf(S[i].z, kn[i], z.z);
                z.w = fmaf(S[i].w, kn[i], z.w);
                y.x = fmaf(S[i].x, qn, y.x);
                y.y = fmaf(S[i].y, qn, y.y);
                y.z = fmaf(S[i].z, qn, y.z);
                y.w = fmaf(S[i].w, qn, y.w);
            }
#pragma unroll
            for (int o = 8; o <= 16; o <<= 1) {
                z.x += __shfl_xor_sync(0xffffffffu, z.x, o);
                z.y += __shfl_xor_sync(0xffffffffu, z.y, o);
                z.z += __shfl_xor_sync(0xffffffffu, z.z, o);
                z.w += __shfl_xor_sync(0xffffffffu, z.w, o);
                y.x += __shfl_xor_sync(0xffffffffu, y.x, o);
                y.y += __shfl_xor_sync(0xffffffffu, y.y, o);
                y.z += __shfl_xor_sync(0xffffffffu, y.z, o);
                y.w += __shfl_xor_sync(0xffffffffu, y.w, o);
            }
            float *rz = red + (rr & 1) * kRed, *ry = rz + 8 * kRecV;
            if (lane < 8) {
                *reinterpret_cast<float4*>(rz + warp * kRecV + c4) = z;
                *reinterpret_cast<float4*>(ry + warp * kRecV + c4) = y;
            }
            __syncthreads();   // also frees qs / ks / vs for the next row
            z = y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float4 p = *reinterpret_cast<const float4*>(rz + i * kRecV + c4);
                z.x += p.x;
                z.y += p.y;
                z.z += p.z;
                z.w += p.w;
            }
            const float4 u = make_float4(w * (v.x - z.x), w * (v.y - z.y), w * (v.z - z.z), w * (v.w - z.w));
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                S[i].x = fmaf(kn[i], u.x, S[i].x);
                S[i].y = fmaf(kn[i], u.y, S[i].y);
                S[i].z = fmaf(kn[i], u.z, S[i].z);
                S[i].w = fmaf(kn[i], u.w, S[i].w);
            }
            if (warp == 0 && lane < 8 && colv) {
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    const float4 p = *reinterpret_cast<const float4*>(ry + i * kRecV + c4);
                    y.x += p.x;
                    y.y += p.y;
                    y.z += p.z;
                    y.w += p.w;
                }
                *reinterpret_cast<float4*>(a.o + (long)row * a.ldo + h * V8 + v0 + c4) =
                    make_float4(fmaf(kq, u.x, y.x), fmaf(kq, u.y, y.y), fmaf(kq, u.z, y.z), fmaf(kq, u.w, y.w));
            }
            continue;
        }
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int n = ng + 32 * i;
            const float kw = ks[n] * w, qn = qs[n];
            S[i].x = fmaf(d, S[i].x, kw * v.x);
            S[i].y = fmaf(d, S[i].y, kw * v.y);
            S[i].z = fmaf(d, S[i].z, kw * v.z);
            S[i].w = fmaf(d, S[i].w, kw * v.w);
            y.x = fmaf(S[i].x, qn, y.x);
            y.y = fmaf(S[i].y, qn, y.y);
            y.z = fmaf(S[i].z, qn, y.z);
            y.w = fmaf(S[i].w, qn, y.w);
        }
#pragma unroll
        for (int o = 8; o <= 16; o <<= 1) {
            y.x += __shfl_xor_sync(0xffffffffu, y.x, o);
            y.y += __shfl_xor_sync(0xffffffffu, y.y, o);
            y.z += __shfl_xor_sync(0xffffffffu, y.z, o);
            y.w += __shfl_xor_sync(0xffffffffu, y.w, o);
        }
        float* rb = red + (rr & 1) * kRed;
        if (lane < 8) *reinterpret_cast<float4*>(rb + warp * kRecV + c4) = y;
        const float vt = t < kRecV ? vs[t] : 0.f;
        __syncthreads();   // also frees qs / ks / vs for the next row
        if (t < kRecV && v0 + t < V8) {
            float s = Dh * vt;
#pragma unroll
            for (int i = 0; i < 8; ++i) s += rb[i * kRecV + t];
            a.o[(long)row * a.ldo + h * V8 + v0 + t] = s;
        }
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int n = ng + 32 * i;
        if (colv && n < N) *reinterpret_cast<float4*>(Sg + (long)n * V8) = S[i];
    }
}

// ---------------------------------------------------------------------------------------------- chunks of 64 tokens
constexpr int kChunk = 64;
constexpr int kPRow = kChunk * 2 + 16;   // bytes of a row of scores in shared memory (odd multiple of 16)
constexpr float kLog2e = 1.4426950408889634f;

struct ChunkSmem {
    int qrow, k_off, v_off, buf, vw_off, s_off, p_off, f_off, total;
    __host__ __device__ ChunkSmem(int N, int VT, int nbuf) {   // VT: state columns per CTA
        const int NP = pad16(N), kVRow = VT * 2 + 16;
        qrow = NP * 2 + 16;
        k_off = kChunk * qrow;
        v_off = 2 * kChunk * qrow;
        buf = v_off + kChunk * kVRow;              // one buffer: q, k, v
        vw_off = nbuf * buf;                       // weighted values, high and remainder
        s_off = vw_off + 2 * kChunk * kVRow;       // state, high and remainder
        p_off = s_off + 2 * NP * kVRow;            // decayed scores, high and remainder
        f_off = p_off + 2 * kChunk * kPRow;        // cumulative log decay, weights
        total = f_off + 2 * 3 * kChunk * 4;
    }
};

// NTW: 16-row state tiles per warp; VT: state columns per CTA (64 or 32).
template <int NTW, int VT>
__global__ void __launch_bounds__(256) recurrence_chunk_kernel(const RecurrenceArgs a, const Rows r, int nbuf) {
    extern __shared__ __align__(16) unsigned char smem[];
    constexpr int kVRow = VT * 2 + 16, NJ = VT / 16;   // NJ: 8-column output tiles per warp
    const ChunkSmem L(a.N, VT, nbuf);
    const int NP = pad16(a.N), N8 = pad8(a.N), V8 = pad8(a.V);
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, q4 = lane & 3;
    const int h = blockIdx.y, v0 = blockIdx.x * VT, grp = h / (a.heads / a.groups);
    const uint32_t sb = smem_u32(smem);
    float* dec = reinterpret_cast<float*>(smem + L.f_off);   // [2][cumulative log2 decay, weight, weight left at the end][chunk]
    const int nchunks = (r.T + kChunk - 1) / kChunk;
    const bf16* qg = static_cast<const bf16*>(a.q) + grp * N8;
    const bf16* kg = static_cast<const bf16*>(a.k) + grp * N8;
    const bf16* vg = static_cast<const bf16*>(a.v) + h * V8 + v0;
    pdl_wait();

    const RowWalk walk(t, 256, NP / 8);
    auto issue = [&](int ch, int buf) {
        const uint32_t base = sb + buf * L.buf;
        for (RowWalk w = walk; w.row < kChunk; w.next()) {
            const int col = w.col * 8, tok = ch * kChunk + w.row;
            const bool ok = tok < r.T && col < N8;
            cp_async16z(base + w.row * L.qrow + col * 2, ok ? qg + (long)tok * a.ldq + col : qg, ok);
            cp_async16z(base + L.k_off + w.row * L.qrow + col * 2, ok ? kg + (long)tok * a.ldk + col : kg, ok);
        }
        for (int i = t; i < kChunk * (VT / 8); i += 256) {
            const int row = i / (VT / 8), col = (i % (VT / 8)) * 8, tok = ch * kChunk + row;
            const bool ok = tok < r.T && v0 + col < V8;
            cp_async16z(base + L.v_off + row * kVRow + col * 2, ok ? vg + (long)tok * a.ldv + col : vg, ok);
        }
        cp_async_commit();
    };

    // state fragments: rows 16 * (i * 8 + warp) .., columns 8 * j ..
    float S[NTW][VT / 8][4];
    float* Sg = a.S + (((long)r.slot * a.heads + h) * a.N) * V8 + v0;
    auto state_to_smem = [&] {
#pragma unroll
        for (int i = 0; i < NTW; ++i) {
            const int n0 = 16 * (i * 8 + warp);
            if (n0 >= NP) continue;
#pragma unroll
            for (int j = 0; j < VT / 8; ++j)
#pragma unroll
                for (int p = 0; p < 2; ++p) {
                    uint32_t hi, lo;
                    split_bf16(S[i][j][2 * p], S[i][j][2 * p + 1], hi, lo);
                    const int off = L.s_off + (n0 + g + 8 * p) * kVRow + (8 * j + 2 * q4) * 2;
                    *reinterpret_cast<uint32_t*>(smem + off) = hi;
                    *reinterpret_cast<uint32_t*>(smem + off + NP * kVRow) = lo;
                }
        }
    };
    // warp 0 keeps the decays one chunk ahead: the loads of the next chunk are in flight during this one
    float l[2], w[2];
    auto load_decay = [&](int ch) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int tok = ch * kChunk + 2 * lane + i;
            const bool ok = tok < r.T;   // rows past the end: no decay, no weight
            l[i] = !ok ? 0.f : a.log_decay ? a.log_decay[(long)tok * a.heads + h] : a.head_log_decay[h];
            w[i] = !ok ? 0.f : a.log_decay ? a.weight[(long)tok * a.heads + h] : a.const_weight;
        }
    };
    auto store_decay = [&](int buf) {
        const float l0 = l[0] * kLog2e, pair = l0 + l[1] * kLog2e;
        float s = pair;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s += up;
        }
        const float first = (s - pair) + l0, total = __shfl_sync(0xffffffffu, s, 31);
        float* cum = dec + buf * 3 * kChunk;
        *reinterpret_cast<float2*>(cum + 2 * lane) = make_float2(first, s);
        *reinterpret_cast<float2*>(cum + kChunk + 2 * lane) = make_float2(w[0], w[1]);
        *reinterpret_cast<float2*>(cum + 2 * kChunk + 2 * lane) = make_float2(exp2_fast(total - first) * w[0], exp2_fast(total - s) * w[1]);
    };
    issue(0, 0);
    if (warp == 0) {
        load_decay(0);
        store_decay(0);
    }
#pragma unroll
    for (int i = 0; i < NTW; ++i)
#pragma unroll
        for (int j = 0; j < VT / 8; ++j)
#pragma unroll
            for (int p = 0; p < 2; ++p) {
                const int n = 16 * (i * 8 + warp) + g + 8 * p, v = 8 * j + 2 * q4;
                float2 s = make_float2(0.f, 0.f);
                if (r.pos0 > 0 && n < a.N && v0 + v < V8) s = *reinterpret_cast<const float2*>(Sg + (long)n * V8 + v);
                S[i][j][2 * p] = s.x;
                S[i][j][2 * p + 1] = s.y;
            }
    state_to_smem();

    for (int ch = 0; ch < nchunks; ++ch) {
        const int buf = nbuf == 2 ? ch & 1 : 0;
        const uint32_t qb = sb + buf * L.buf, kb = qb + L.k_off, vb = qb + L.v_off;
        cp_async_wait<0>();
        __syncthreads();   // operands, state copy and decays are in shared memory
        if (nbuf == 2 && ch + 1 < nchunks) issue(ch + 1, buf ^ 1);
        if (warp == 0) load_decay(ch + 1);
        const float *cum = dec + (ch & 1) * 3 * kChunk, *wt = cum + kChunk, *left = wt + kChunk;
        const float total = cum[kChunk - 1];
        const int r0 = 16 * (warp & 3), c0 = 32 * (warp >> 2);   // score columns; output columns start at
        const int o0 = (VT / 2) * (warp >> 2);
        const float cg0 = cum[r0 + g], cg1 = cum[r0 + g + 8];

        // scores q k^T and inter-chunk part q S, both over the N dimension
        float sc[4][4] = {}, out[NJ][4] = {};
#pragma unroll 2
        for (int k0 = 0; k0 < NP; k0 += 16) {
            uint32_t fa[4];
            ldsm4(qb + (r0 + (lane & 15)) * L.qrow + (k0 + (lane >> 4) * 8) * 2, fa);
#pragma unroll
            for (int jj = 0; jj < 2; ++jj) {
                if (c0 + 16 * jj <= r0 + 15) {
                    uint32_t fb[4];   // two 8-token tiles of k rows: (k low, k high) each
                    ldsm4(kb + (c0 + 16 * jj + (lane & 7) + (lane >> 4) * 8) * L.qrow + (k0 + ((lane >> 3) & 1) * 8) * 2, fb);
                    mma_bf16(sc[2 * jj], fa[0], fa[1], fa[2], fa[3], fb[0], fb[1]);
                    mma_bf16(sc[2 * jj + 1], fa[0], fa[1], fa[2], fa[3], fb[2], fb[3]);
                }
            }
#pragma unroll
            for (int jj = 0; jj < NJ / 2; ++jj)
#pragma unroll
                for (int part = 0; part < 2; ++part) {
                    uint32_t fs[4];
                    ldsm4t(sb + L.s_off + part * NP * kVRow + (k0 + (lane & 15)) * kVRow + (o0 + 16 * jj + (lane >> 4) * 8) * 2, fs);
                    mma_bf16(out[2 * jj], fa[0], fa[1], fa[2], fa[3], fs[0], fs[1]);
                    mma_bf16(out[2 * jj + 1], fa[0], fa[1], fa[2], fa[3], fs[2], fs[3]);
                }
        }
        const float e0 = exp2_fast(cg0), e1 = exp2_fast(cg1);
#pragma unroll
        for (int j = 0; j < NJ; ++j) { out[j][0] *= e0; out[j][1] *= e0; out[j][2] *= e1; out[j][3] *= e1; }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int col = c0 + 8 * j + 2 * q4, ra = r0 + g, rb = ra + 8;
            const float cc0 = cum[col], cc1 = cum[col + 1], w0 = wt[col], w1 = wt[col + 1];
            const float p0 = col <= ra ? sc[j][0] * exp2_fast(cg0 - cc0) * w0 : 0.f, p1 = col + 1 <= ra ? sc[j][1] * exp2_fast(cg0 - cc1) * w1 : 0.f;
            const float p2 = col <= rb ? sc[j][2] * exp2_fast(cg1 - cc0) * w0 : 0.f, p3 = col + 1 <= rb ? sc[j][3] * exp2_fast(cg1 - cc1) * w1 : 0.f;
            uint32_t hi, lo;
            unsigned char* pd = smem + L.p_off + ra * kPRow + col * 2;
            split_bf16(p0, p1, hi, lo);
            *reinterpret_cast<uint32_t*>(pd) = hi;
            *reinterpret_cast<uint32_t*>(pd + kChunk * kPRow) = lo;
            split_bf16(p2, p3, hi, lo);
            *reinterpret_cast<uint32_t*>(pd + 8 * kPRow) = hi;
            *reinterpret_cast<uint32_t*>(pd + 8 * kPRow + kChunk * kPRow) = lo;
        }
        // values weighted by what is left of them at the end of the chunk
        for (int i = t; i < kChunk * VT / 2; i += 256) {
            const int row = i / (VT / 2), col = (i % (VT / 2)) * 2;
            const uint32_t vv = *reinterpret_cast<const uint32_t*>(smem + buf * L.buf + L.v_off + row * kVRow + col * 2);
            const float f = left[row];
            uint32_t hi, lo;
            split_bf16(__uint_as_float(vv << 16) * f, __uint_as_float(vv & 0xFFFF0000u) * f, hi, lo);
            *reinterpret_cast<uint32_t*>(smem + L.vw_off + row * kVRow + col * 2) = hi;
            *reinterpret_cast<uint32_t*>(smem + L.vw_off + (kChunk + row) * kVRow + col * 2) = lo;
        }
        if (warp == 0) store_decay((ch + 1) & 1);
        __syncthreads();   // scores and weighted values written, old state copy read

        // within the chunk: out += P v
        for (int k0 = 0; k0 <= r0; k0 += 16) {
            uint32_t ph[4], pl[4];
            const uint32_t pa = sb + L.p_off + (r0 + (lane & 15)) * kPRow + (k0 + (lane >> 4) * 8) * 2;
            ldsm4(pa, ph);
            ldsm4(pa + kChunk * kPRow, pl);
#pragma unroll
            for (int jj = 0; jj < NJ / 2; ++jj) {
                uint32_t fv[4];
                ldsm4t(vb + (k0 + (lane & 15)) * kVRow + (o0 + 16 * jj + (lane >> 4) * 8) * 2, fv);
                mma_bf16(out[2 * jj], ph[0], ph[1], ph[2], ph[3], fv[0], fv[1]);
                mma_bf16(out[2 * jj], pl[0], pl[1], pl[2], pl[3], fv[0], fv[1]);
                mma_bf16(out[2 * jj + 1], ph[0], ph[1], ph[2], ph[3], fv[2], fv[3]);
                mma_bf16(out[2 * jj + 1], pl[0], pl[1], pl[2], pl[3], fv[2], fv[3]);
            }
        }
        const float Dh = a.D ? a.D[h] : 0.f;
#pragma unroll
        for (int j = 0; j < NJ; ++j)
#pragma unroll
            for (int p = 0; p < 2; ++p) {
                const int row = r0 + g + 8 * p, col = o0 + 8 * j + 2 * q4, tok = ch * kChunk + row;
                if (tok < r.T && v0 + col < V8) {
                    float2 o2 = make_float2(out[j][2 * p], out[j][2 * p + 1]);
                    if (a.D) {
                        const uint32_t vv = *reinterpret_cast<const uint32_t*>(smem + buf * L.buf + L.v_off + row * kVRow + col * 2);
                        o2.x = fmaf(Dh, __uint_as_float(vv << 16), o2.x);
                        o2.y = fmaf(Dh, __uint_as_float(vv & 0xFFFF0000u), o2.y);
                    }
                    *reinterpret_cast<float2*>(a.o + (long)tok * a.ldo + h * V8 + v0 + col) = o2;
                }
            }
        // state: S = exp(total) S + k^T (weighted v)
        const float et = exp2_fast(total);
#pragma unroll
        for (int i = 0; i < NTW; ++i) {
            const int n0 = 16 * (i * 8 + warp);
            if (n0 >= NP) continue;
#pragma unroll
            for (int j = 0; j < VT / 8; ++j)
#pragma unroll
                for (int p = 0; p < 4; ++p) S[i][j][p] *= et;
#pragma unroll
            for (int k0 = 0; k0 < kChunk; k0 += 16) {
                uint32_t fk[4];   // k^T: row n, column token
                ldsm4t(kb + (k0 + (lane & 7) + (lane >> 4) * 8) * L.qrow + (n0 + ((lane >> 3) & 1) * 8) * 2, fk);
#pragma unroll
                for (int jj = 0; jj < VT / 16; ++jj)
#pragma unroll
                    for (int part = 0; part < 2; ++part) {
                        uint32_t fv[4];
                        ldsm4t(sb + L.vw_off + (part * kChunk + k0 + (lane & 15)) * kVRow + (16 * jj + (lane >> 4) * 8) * 2, fv);
                        mma_bf16(S[i][2 * jj], fk[0], fk[1], fk[2], fk[3], fv[0], fv[1]);
                        mma_bf16(S[i][2 * jj + 1], fk[0], fk[1], fk[2], fk[3], fv[2], fv[3]);
                    }
            }
        }
        state_to_smem();
        if (nbuf == 1) {
            __syncthreads();
            if (ch + 1 < nchunks) issue(ch + 1, 0);
        }
    }
#pragma unroll
    for (int i = 0; i < NTW; ++i)
#pragma unroll
        for (int j = 0; j < VT / 8; ++j)
#pragma unroll
            for (int p = 0; p < 2; ++p) {
                const int n = 16 * (i * 8 + warp) + g + 8 * p, v = 8 * j + 2 * q4;
                if (n < a.N && v0 + v < V8)
                    *reinterpret_cast<float2*>(Sg + (long)n * V8 + v) = make_float2(S[i][j][2 * p], S[i][j][2 * p + 1]);
            }
}

}  // namespace lm
}  // namespace bw
