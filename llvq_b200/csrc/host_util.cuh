// Host-side plumbing of a C ABI translation unit: the error text of the last failed call, the launch
// counter, the programmatic-dependent launch and the dynamic shared-memory opt-in. Every shared object
// includes it in exactly one source, so each keeps its own error text and counter.
#pragma once
#include <cuda_runtime.h>

#include <atomic>
#include <cstdarg>
#include <cstdint>
#include <cstdio>
#include <map>
#include <mutex>
#include <string>
#include <utility>

namespace {

// the status values of include/llvq_b200.h and include/llvq_dense.h
constexpr int kStatusOk = 0, kStatusInvalid = -1, kStatusCuda = -2, kStatusUnsupported = -5;

thread_local std::string g_error;
std::atomic<uint64_t> g_launches{0};

int fail(int code, const char* fmt, ...) {
    char buf[512];
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(buf, sizeof buf, fmt, ap);
    va_end(ap);
    g_error = buf;
    return code;
}

#define CUDA_TRY(expr)                                                                          \
    do {                                                                                        \
        cudaError_t e_ = (expr);                                                                \
        if (e_ != cudaSuccess)                                                                  \
            return fail(kStatusCuda, "%s failed: %s (%s:%d)", #expr, cudaGetErrorString(e_), \
                        __FILE__, __LINE__);                                                    \
    } while (0)

// Launch with programmatic stream serialisation (see llvq_runtime_set_overlap): the kernel may be scheduled
// while the previous kernel of the stream is still running; it orders itself behind that kernel with
// griddepcontrol.wait before it touches memory (llvq_dependent_enter, or the GEMV's own placement of the wait).
std::atomic<int> g_overlap_ops{1};
template <typename... KArgs, typename... Args>
cudaError_t launch_dep(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, Args&&... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = g_overlap_ops.load(std::memory_order_relaxed) ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kern, std::forward<Args>(args)...);
}

// cudaFuncAttributeMaxDynamicSharedMemorySize is a per-device setting: remember, per (device, kernel),
// the largest size configured so far, so that a second runtime on another GPU raises it again.
std::mutex g_smem_mu;
std::map<std::pair<int, const void*>, size_t> g_smem_configured;

int ensure_dyn_smem(const void* func, size_t bytes) {
    int dev = 0;
    CUDA_TRY(cudaGetDevice(&dev));
    std::lock_guard<std::mutex> lock(g_smem_mu);
    size_t& have = g_smem_configured[{dev, func}];
    if (bytes > have) {
        CUDA_TRY(cudaFuncSetAttribute(func, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
        have = bytes;
    }
    return kStatusOk;
}

}  // namespace
