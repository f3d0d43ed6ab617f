// Host plumbing linked into both libraries: error messages, the device's SM count, the chained-launch scope.
#include <atomic>
#include <cstdarg>
#include <cstdio>
#include <cstdlib>

#include "common.cuh"

namespace sk {

static thread_local char g_err[512] = "";
static thread_local int g_pdl_depth = 0;

bool pdl_chain_active() {
    static const bool off = getenv("SOCKET_B200_NO_PDL") != nullptr;   // debugging aid: launch the step's kernels unchained
    return g_pdl_depth > 0 && !off;
}
PdlChain::PdlChain() { ++g_pdl_depth; }
PdlChain::~PdlChain() { --g_pdl_depth; }

int fail(int status, const char* fmt, ...) {
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(g_err, sizeof(g_err), fmt, ap);
    va_end(ap);
    return status;
}

int sm_count() {
    constexpr int MAX_DEV = 64;
    static std::atomic<int> cached[MAX_DEV];
    int dev = -1;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= MAX_DEV) {
        cudaGetLastError();   // a size query without a device is not an error of the next launch
        return 148;
    }
    int n = cached[dev].load(std::memory_order_relaxed);
    if (n > 0) return n;
    if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) {
        cudaGetLastError();
        return 148;
    }
    cached[dev].store(n, std::memory_order_relaxed);
    return n;
}

int check_launch(const char* what) {
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return fail(SK_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
    return SK_OK;
}

const char* last_error() { return g_err; }

const char* status_string(int status) {
    switch (status) {
        case SK_OK: return "ok";
        case SK_ERR_INVALID_ARGUMENT: return "invalid argument";
        case SK_ERR_UNSUPPORTED: return "unsupported shape or dtype";
        case SK_ERR_MISALIGNED: return "misaligned pointer or stride";
        case SK_ERR_WORKSPACE: return "workspace too small";
        case SK_ERR_CUDA: return "CUDA runtime error";
        default: return "unknown status";
    }
}

}  // namespace sk
