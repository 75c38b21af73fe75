// Per-device facts and kernel attributes, cached.
#include "common.cuh"
#include <map>
#include <mutex>

namespace mk {

void ensure_dynamic_smem(const void* func, size_t bytes) {
    if (bytes <= 32 * 1024) return;  // 48 KB need no opt-in, the kernel's static shared memory included
    static std::mutex mu;
    static std::map<std::pair<const void*, int>, size_t> done;
    int dev = 0;
    MK_CUDA(cudaGetDevice(&dev));
    std::lock_guard<std::mutex> lock(mu);
    size_t& have = done[{func, dev}];
    if (have >= bytes) return;
    MK_CUDA(cudaFuncSetAttribute(func, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
    have = bytes;
}

int device_sm_count() {
    static std::mutex mu;
    static std::map<int, int> cached;
    int dev = 0;
    MK_CUDA(cudaGetDevice(&dev));
    std::lock_guard<std::mutex> lock(mu);
    int& n = cached[dev];
    if (n == 0) MK_CUDA(cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev));
    return n;
}

}  // namespace mk
