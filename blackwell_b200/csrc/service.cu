// Library-wide service state: launch accounting, the programmatic-dependent-launch switch and the device status word
// that bounded waits report through.
#include <cuda_runtime.h>

#include <atomic>
#include <mutex>

#include "../../include/blackwell_b200.h"
#include "host_util.h"

namespace bw {

static std::atomic<long long> g_launches{0};
void count_launch(int n) { g_launches.fetch_add(n, std::memory_order_relaxed); }

static std::atomic<int> g_pdl{1};
bool pdl_enabled() { return g_pdl.load() != 0; }
void set_pdl(int on) { g_pdl = on; }

// One status word per device for the whole library: kernels that give up on a bounded wait store a code here.
static __device__ int g_status_word = 0;
int* status_word_ptr() {
    static int* ptr[kMaxDevices] = {nullptr};
    static std::mutex mu;
    std::lock_guard<std::mutex> lk(mu);
    const int dev = current_device();
    if (!ptr[dev]) {
        int* p = nullptr;
        if (cudaGetSymbolAddress(reinterpret_cast<void**>(&p), g_status_word) != cudaSuccess) return nullptr;
        ptr[dev] = p;
    }
    return ptr[dev];
}

}  // namespace bw

extern "C" int bw_device_status(int* status_out) {
    int* p = bw::status_word_ptr();
    if (!p) return cudaErrorInitializationError;
    int v = 0;
    cudaError_t e = cudaMemcpy(&v, p, sizeof(int), cudaMemcpyDeviceToHost);
    if (e != cudaSuccess) return e;
    if (v != 0) {
        const int zero = 0;
        e = cudaMemcpy(p, &zero, sizeof(int), cudaMemcpyHostToDevice);
    }
    if (status_out) *status_out = v;
    return e;
}

extern "C" long long bw_launch_count(int reset) {
    return reset ? bw::g_launches.exchange(0) : bw::g_launches.load();
}

extern "C" int bw_version(void) { return 100; }
