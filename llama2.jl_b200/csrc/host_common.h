// Host-side helpers shared by the CUDA translation units of the library (api.cu, stack.cu): the per-thread error text,
// the status macros, kernel launches with their attributes, and the tensor-map encoder of the driver.
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>

#include <cstdlib>
#include <cstring>
#include <string>

#include "../../include/llama2_b200.h"

// Records the text of a failure for l2b_last_error_string and returns `code` (defined in api.cu).
int32_t fail(int32_t code, const std::string& msg);

#define CU(call)                                                                                         \
    do {                                                                                                 \
        cudaError_t e_ = (call);                                                                         \
        if (e_ != cudaSuccess) {                                                                         \
            (void)cudaGetLastError();                                                                    \
            return fail(e_ == cudaErrorMemoryAllocation ? L2B_ERR_OOM : L2B_ERR_CUDA,                    \
                        std::string(#call) + ": " + cudaGetErrorString(e_) + " (" + __FILE__ + ":" + std::to_string(__LINE__) + ")"); \
        }                                                                                                \
    } while (0)

#define L2B_TRY(expr)              \
    do {                           \
        int32_t s_ = (expr);       \
        if (s_ != L2B_OK) return s_; \
    } while (0)

struct DeviceInfo {
    int sms = 148;
    int max_smem_optin = 227 * 1024;
};

static inline int32_t query_device(DeviceInfo& di) {
    int dev = 0;
    CU(cudaGetDevice(&dev));
    CU(cudaDeviceGetAttribute(&di.sms, cudaDevAttrMultiProcessorCount, dev));
    CU(cudaDeviceGetAttribute(&di.max_smem_optin, cudaDevAttrMaxSharedMemoryPerBlockOptin, dev));
    return L2B_OK;
}

// pdl: launched with a programmatic dependency on the previous kernel of the stream.
// cluster > 1: the grid is launched as thread-block clusters of that many consecutive blocks.
template <typename Kernel, typename... Args>
static cudaError_t launch_kernel_args(Kernel k, dim3 grid, dim3 block, size_t smem, cudaStream_t st, bool pdl, int cluster, const Args&... args) {
    cudaLaunchConfig_t cfg;
    memset(&cfg, 0, sizeof(cfg));
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (pdl) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n].val.programmaticStreamSerializationAllowed = 1;
        ++n;
    }
    if (cluster > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = (unsigned)cluster;
        attr[n].val.clusterDim.y = 1;
        attr[n].val.clusterDim.z = 1;
        ++n;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    return cudaLaunchKernelEx(&cfg, k, args...);
}
template <typename Kernel, typename Params>
static cudaError_t launch_kernel(Kernel k, dim3 grid, dim3 block, size_t smem, cudaStream_t st, bool pdl, const Params& prm, int cluster = 1) {
    return launch_kernel_args(k, grid, block, smem, st, pdl, cluster, prm);
}

static inline long env_long(const char* name, long dflt) {
    const char* v = getenv(name);
    return v && *v ? atol(v) : dflt;
}

// cuTensorMapEncodeTiled comes from the driver; the library links the runtime only, so the entry point is looked up.
typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                  const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static inline EncodeTiledFn encode_tiled_fn() {
    static EncodeTiledFn fn = [] {
        void* f = nullptr;
        cudaDriverEntryPointQueryResult qr;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &f, cudaEnableDefault, &qr) != cudaSuccess || qr != cudaDriverEntryPointSuccess) {
            (void)cudaGetLastError();
            f = nullptr;
        }
        return (EncodeTiledFn)f;
    }();
    return fn;
}
