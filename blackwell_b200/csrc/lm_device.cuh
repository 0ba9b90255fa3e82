// Device helpers of the bfloat16 kernels: typed loads and stores, warp-level bf16 MMA, ldmatrix, cp.async.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

namespace bw {
namespace lm {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename A> __device__ __forceinline__ A from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}
// (x, y) -> packed bf16 high parts and packed bf16 remainders: together 16 significant bits.
__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(x, y);
    lo = pack_bf16(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xFFFF0000u));
}

// 16 bytes, or zeros when !valid (src must still be a readable address)
__device__ __forceinline__ void cp_async16z(uint32_t dst, const void* src, bool valid) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
// D(16x8) += A(16x16) B(16x8), bf16 operands, fp32 accumulators.  Thread (g = lane / 4, t = lane % 4): a0 row g, a1 row
// g + 8 (columns 2t, 2t+1), a2 / a3 the same rows, columns 2t+8, 2t+9; b0 / b1 rows 2t, 2t+1 / 2t+8, 2t+9 of column g;
// c0, c1 row g, c2, c3 row g + 8, columns 2t, 2t+1.
__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// 2^x by the hardware instruction (subnormal results become zero).
__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// Walks the elements t, t + threads, t + 2 * threads, ... of a [rows][cols] array without a division per step.
struct RowWalk {
    int row, col, drow, dcol, cols;
    __device__ __forceinline__ RowWalk(int t, int threads, int cols_)
        : row(t / cols_), col(t % cols_), drow(threads / cols_), dcol(threads % cols_), cols(cols_) {}
    __device__ __forceinline__ void next() {
        row += drow;
        col += dcol;
        if (col >= cols) { col -= cols; ++row; }
    }
};

// Bulk copy of one row (16-byte aligned on both sides, size a multiple of 16), counted in bytes on an mbarrier.
__device__ __forceinline__ void bulk_row(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                 ::"r"(dst), "l"(src), "r"(bytes), "r"(bar)
                 : "memory");
}
// Waits for a copy phase; after a wait that gave up (status word set) the thread does not wait again, so that every thread
// still meets its block's barriers and the kernel ends.
struct CopyWait {
    int* status;
    bool dead = false;
    __device__ __forceinline__ void operator()(uint32_t bar, uint32_t parity) {
        if (!dead && !mbar_wait(bar, parity)) {
            dead = true;
            if (status) *status = kStatusMbarTimeout;
        }
    }
};
// Zeroes `bytes` (a multiple of 16) of shared memory that bulk copies will fill: rows and columns they do not cover stay zero.
__device__ __forceinline__ void zero_smem(unsigned char* p, int bytes, int t, int threads) {
    for (int i = t * 16; i < bytes; i += threads * 16) *reinterpret_cast<uint4*>(p + i) = make_uint4(0, 0, 0, 0);
}

// Shared memory of another block of the cluster, and the cluster's barrier.
__device__ __forceinline__ float ld_dsmem(uint32_t addr, uint32_t rank) {
    uint32_t ra;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(ra) : "r"(addr), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(ra) : "memory");
    return v;
}
__device__ __forceinline__ void cluster_sync_all() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}

// Sum over a block of up to 1024 threads; every thread gets the total.  `buf`: 32 floats of shared memory.
__device__ __forceinline__ float block_sum(float v, float* buf) {
    v = warp_sum(v);
    const int warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    if ((threadIdx.x & 31) == 0) buf[warp] = v;
    __syncthreads();
    float t = 0.f;
    for (int i = 0; i < nw; ++i) t += buf[i];
    __syncthreads();
    return t;
}

}  // namespace lm
}  // namespace bw
