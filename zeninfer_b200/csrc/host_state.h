// The host-side pieces the library's translation units share: the weight handle and the entry guard of the C-ABI calls.
#pragma once
#include <cuda_runtime.h>

#include <cstdint>
#include <mutex>
#include <string>

struct zen_cuda_weights {
    int format{};
    size_t rows{}, cols{};
    uint32_t nb{}, nbp{};     // blocks per row, padded to 8
    void* plane[4]{};         // format-specific planes (see repack.cuh)
    void* d_tile_maps{};      // Q8_0 rows of several K segments: zk::GemvTileMaps in device memory (see make_tile_maps), else null
    int kernel_format{};      // what the decode kernel is instantiated for: the format, or zk::kFormatQ6KCodes for Q6_K with unpacked codes
    // Two-digit planes under one scale per 256 weights (gemm_groups.cuh), built at the tensor's first many-row product and
    // kept: wh, wl [rows][cols] int8, units [rows][cols / 256] fp32.
    mutable void* g_hi{};
    mutable void* g_lo{};
    mutable float* g_unit{};
    mutable size_t g_bytes{};
    size_t device_bytes{};
    size_t raw_bytes{};
};

namespace zk_host {

// One C-ABI call: holds the backend's lock, makes the backend ready (ok), and carries what a launch needs.
struct Entry {
    std::lock_guard<std::mutex> lock;
    bool ok;
    cudaStream_t stream;
    int* d_error;             // the kernels' error word
    void* encode_tiled;       // cuTensorMapEncodeTiled
    int sm_count;
    size_t smem_optin;
    bool pdl;                 // programmatic dependent launch
    explicit Entry(void* stream_arg);
    int fail(const std::string& why);                       // records the message, returns 0
    int leave(cudaError_t launch_result, const char* what); // counts the launch, returns 1 or 0
};

bool set_dense_wait_budget(long long cycles);   // zen_cuda_dense.cu's copy of the bounded-wait budget

}  // namespace zk_host
