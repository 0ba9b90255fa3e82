// Host side of the bfloat16 linear kernels: routing by row count, tensor maps, launch shapes.
#include <cuda_runtime.h>

#include <atomic>
#include <mutex>

#include "../../include/blackwell_b200.h"
#include "host_util.h"
#include "linear_bf16.cuh"
#include "tensor_map.h"

namespace bw {
namespace lm {
namespace {

static_assert(kTcK == kMapCols, "a K block is one box");

template <typename F>
cudaError_t allow_smem(F kern, std::once_flag (&once)[kMaxDevices], int bytes) {
    cudaError_t e = cudaSuccess;
    std::call_once(once[current_device()], [&] { e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes); });
    return e;
}

int stream_xs_stride(int ldw) {
    const int nkb = (ldw + 31) / 32;
    return nkb * 64 + (nkb % 2 == 0 ? 64 : 0);   // odd multiple of 64 bytes: conflict-free fragment reads
}
int stream_smem(int T, int ldw) { return kStreamWarps * 8 * 16 * 4 + T * stream_xs_stride(ldw); }

cudaError_t launch_stream(const LinearArgs& a, cudaStream_t st) {
    static std::once_flag once[kMaxDevices];
    cudaError_t e = allow_smem(linear_stream_kernel, once, kMaxDynSmem);
    if (e != cudaSuccess) return e;
    const int smem = stream_smem(a.T, (int)a.ldw), tiles = (a.N + 15) / 16;
    const int per_sm = smem > 110 * 1024 ? 1 : smem > 72 * 1024 ? 2 : 3;
    const int grid = std::min(tiles, sm_count(current_device()) * per_sm);
    e = launch_pdl(linear_stream_kernel, dim3(grid), dim3(kStreamWarps * 32), smem, st, a, stream_xs_stride((int)a.ldw));
    count_launch(1);
    return e;
}

template <int NT, bool SPLIT>
cudaError_t launch_tc(const LinearArgs& a, int ksplit, cudaStream_t st) {
    static std::once_flag once[kMaxDevices];
    auto kern = linear_tc_kernel<NT, SPLIT>;
    const int smem = tc_smem_bytes(NT, SPLIT);
    static_assert(tc_smem_bytes(NT, SPLIT) <= kMaxDynSmem, "shared memory");
    cudaError_t e = allow_smem(kern, once, smem);
    if (e != cudaSuccess) return e;
    if (!encode_fn()) return cudaErrorNotSupported;
    CUtensorMap mw, mx;
    if (!make_map(&mw, a.W, a.K, a.N, a.ldw, kTcRows) || !make_map(&mx, a.x, a.K, a.T, a.ldx, NT)) return cudaErrorInvalidValue;
    const int tiles = ((a.N + kTcRows - 1) / kTcRows) * ((a.T + NT - 1) / NT);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(SPLIT ? tiles * ksplit : std::min(tiles, sm_count(current_device())));
    cfg.blockDim = dim3(kTcThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = ksplit;
    attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = SPLIT ? 2 : 1;   // no cluster in the persistent form
    int* status = status_word_ptr();
    // persistent form: ksplit says whether the weights are too large for L2
    if (!SPLIT) ksplit = (long)a.N * a.K > (24l << 20) && (long)a.N * a.K > (long)a.T * a.K;
    e = cudaLaunchKernelEx(&cfg, kern, mw, mx, a, ksplit, status);
    count_launch(1);
    return e;
}

std::atomic<int> g_stream_max{-1};   // rows up to which the streaming kernel is used; -1: automatic

}  // namespace

void set_linear_stream_max(int rows) { g_stream_max = rows > 0 ? rows - 1 : -1; }

cudaError_t linear(const LinearArgs& a, cudaStream_t st) {
    if (a.T < 1 || a.N < 1 || a.K < 1 || a.ldw % 8 != 0 || a.ldw < a.K || (reinterpret_cast<uintptr_t>(a.W) & 15) ||
        (reinterpret_cast<uintptr_t>(a.x) & 15) || a.ldx < a.K || (a.epi == kEpiSwiglu && a.N % 2 != 0))
        return cudaErrorInvalidValue;
    if (a.f32) {
        const dim3 grid((a.N + 63) / 64, (a.T + 63) / 64);
        cudaError_t e = launch_pdl(linear_f32_kernel, grid, dim3(256), 0, st, a);
        count_launch(1);
        return e;
    }
    if (a.ldx % 8 != 0) return cudaErrorInvalidValue;
    // measured borders: the streaming kernel wins on small matrices and few rows (its launch has less to set up)
    const long size = (long)a.N * a.K;
    const int limit = g_stream_max.load();
    const bool stream = limit >= 0 ? a.T <= limit : a.K <= 4096 && ((a.T <= 2 && size <= 25000000) || (a.K <= 2048 && size <= 8000000));
    if (stream && a.T <= 8 && stream_smem(a.T, (int)a.ldw) <= kMaxDynSmem) return launch_stream(a, st);
    // enough tiles for the SMs: persistent tiles of 256 / 128 rows; otherwise the K range is split over a cluster
    const int sms = sm_count(current_device()), rtiles = (a.N + kTcRows - 1) / kTcRows, nk = (a.K + kTcK - 1) / kTcK;
    auto tiles = [&](int nt_) { return rtiles * ((a.T + nt_ - 1) / nt_); };
    if (a.T > 64) {
        if (tiles(256) >= sms) return launch_tc<256, false>(a, 1, st);
        if (a.T > 512 || tiles(128) >= sms / 2) {
            // fewer, larger tiles only when they fill the machine as well as the small ones do
            const long w128 = (long)((tiles(128) + sms - 1) / sms), w64 = (long)((tiles(64) + sms - 1) / sms);
            return 2 * w64 < 2 * w128 + 1 && w64 * 64 < w128 * 128 ? launch_tc<64, false>(a, 1, st) : launch_tc<128, false>(a, 1, st);
        }
    }
    const int ntile = a.T <= 16 ? 16 : a.T <= 32 ? 32 : 64;
    // K split that finishes first: waves of CTAs (two per SM), each its share of the K blocks plus a constant
    int ks = 1;
    long best = 0;
    for (int k = 1; k <= 8 && k <= nk; k *= 2) {
        const long cost = (long)((tiles(ntile) * k + 2 * sms - 1) / (2 * sms)) * ((nk + k - 1) / k + 8);
        if (k == 1 || cost < best) { best = cost; ks = k; }
    }
    return ntile == 16 ? launch_tc<16, true>(a, ks, st) : ntile == 32 ? launch_tc<32, true>(a, ks, st) : launch_tc<64, true>(a, ks, st);
}

}  // namespace lm
}  // namespace bw

extern "C" int bw_linear_bf16(void* y, long ldy, const void* x, long ldx, const uint16_t* W, long ldw, int T, int N, int K,
                              int y_f32, int x_f32, int epilogue, float softcap, void* stream) {
    if (!y || !x || !W || epilogue < 0 || epilogue > 2) return cudaErrorInvalidValue;
    bw::lm::LinearArgs a{};
    a.x = x; a.ldx = ldx; a.W = reinterpret_cast<const bw::lm::bf16*>(W); a.ldw = ldw; a.T = T; a.N = N; a.K = K;
    a.y = y; a.ldy = ldy; a.y_f32 = y_f32; a.split = N; a.epi = epilogue; a.softcap = softcap; a.f32 = x_f32;
    return bw::lm::linear(a, static_cast<cudaStream_t>(stream));
}
