// State every library of the package has exactly one copy of: the sticky device status word, the launch counter
// and the status texts.  Linked into each shared library (build.py), so it must not depend on any kernel.
#include <atomic>

#include "common.cuh"

namespace tbl {

static std::atomic<uint64_t> g_launches{0};
void note_launch(int n) { g_launches.fetch_add(static_cast<uint64_t>(n), std::memory_order_relaxed); }

__device__ int g_device_status = 0;

int* device_status_ptr() {
    static int* cached[64] = {};
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return nullptr;
    if (!cached[dev]) {
        void* p = nullptr;
        if (cudaGetSymbolAddress(&p, g_device_status) != cudaSuccess) return nullptr;
        cached[dev] = static_cast<int*>(p);
    }
    return cached[dev];
}

int read_and_clear_device_status(int* out) {
    int status = 0;
    if (cudaMemcpyFromSymbol(&status, g_device_status, sizeof(int)) != cudaSuccess) return -1;
    if (status != 0) {
        const int zero = 0;
        if (cudaMemcpyToSymbol(g_device_status, &zero, sizeof(int)) != cudaSuccess) return -1;
    }
    *out = status;
    return 0;
}

}  // namespace tbl

using namespace tbl;

extern "C" {

const char* tbl_status_string(int status) {
    switch (status) {
        case TBL_OK: return "ok";
        case TBL_ERR_INVALID_ARG: return "invalid argument (null pointer, non-positive size or bad flag)";
        case TBL_ERR_SHAPE: return "unsupported shape (K must be a multiple of 16, M*N <= INT_MAX, M within the kernel's range)";
        case TBL_ERR_OVERFLOW: return "K too large: int32 accumulation could overflow";
        case TBL_ERR_SCALE: return "weight_scale must be finite and positive";
        case TBL_ERR_BITS: return "activation bits must be in [2,8]";
        case TBL_ERR_ALIGNMENT: return "device pointer must be 16-byte aligned";
        case TBL_ERR_WORKSPACE: return "workspace too small";
        case TBL_ERR_FORMAT: return "edge pack malformed";
        case TBL_ERR_INTEGRITY: return "edge pack integrity trailer missing or digest mismatch";
        case TBL_ERR_CODE: return "packed words contain the reserved code 0b11";
        case TBL_ERR_CUDA: return "CUDA runtime error";
        case TBL_ERR_UNSUPPORTED: return "descriptor mode not implemented";
        default: return "unknown status";
    }
}

uint64_t tbl_launch_count(void) { return g_launches.load(std::memory_order_relaxed); }

int tbl_device_status(void* stream) {
    cudaError_t e = cudaStreamSynchronize(static_cast<cudaStream_t>(stream));
    if (e != cudaSuccess) return TBL_ERR_CUDA;
    int status = 0;
    if (read_and_clear_device_status(&status) != 0) return TBL_ERR_CUDA;
    return status;
}

}  // extern "C"
