// Library core behind the C ABI (include/stark_b200.h): version, status names, device plumbing, the per-device context.
// No exception crosses the boundary and nothing is printed.
#include <mutex>

#include "context.cuh"

namespace sb {

static std::mutex g_ctx_mutex;
static DeviceContext g_ctx[64];

DeviceContext *device_context() {
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return nullptr;
    std::lock_guard<std::mutex> lock(g_ctx_mutex);
    DeviceContext &c = g_ctx[dev];
    if (c.device != dev) {
        uint32_t *word = nullptr;
        if (cudaMalloc(&word, 256) != cudaSuccess) return nullptr;
        if (cudaMemset(word, 0, 256) != cudaSuccess) {
            cudaFree(word);
            return nullptr;
        }
        c.error_word = word;
        c.device = dev;
    }
    return &c;
}

stark_b200_status ensure_buffer(void **buf, size_t *have, size_t want) {
    if (*have >= want && *buf) return STARK_B200_OK;
    if (*buf) cudaFree(*buf);
    *buf = nullptr;
    *have = 0;
    size_t cap = want < 4096 ? 4096 : want;
    SB_CUDA(cudaMalloc(buf, cap));
    *have = cap;
    return STARK_B200_OK;
}

}  // namespace sb

using namespace sb;

extern "C" {

uint32_t stark_b200_abi_version(void) { return STARK_B200_ABI_VERSION; }

const char *stark_b200_status_name(uint32_t status) {
    switch (status) {
        case STARK_B200_OK: return "ok";
        case STARK_B200_INVALID_ARGUMENT: return "invalid_argument";
        case STARK_B200_ABI_MISMATCH: return "abi_mismatch";
        case STARK_B200_CONTEXT_LIMIT: return "context_limit";
        case STARK_B200_CANCELLED: return "cancelled";
        case STARK_B200_UNSUPPORTED: return "unsupported";
        case STARK_B200_OUT_OF_MEMORY: return "out_of_memory";
        case STARK_B200_IO_FAILURE: return "io_failure";
        case STARK_B200_DEVICE_FAILURE: return "device_failure";
        case STARK_B200_RELOAD_REQUIRED: return "reload_required";
        case STARK_B200_BUSY: return "busy";
        case STARK_B200_INVALID_STATE: return "invalid_state";
        default: return "unknown";
    }
}

const char *stark_b200_last_cuda_error(void) { return cudaGetErrorName(last_cuda_error()); }

stark_b200_status stark_b200_device_count(int32_t *out_count) {
    if (!out_count) return STARK_B200_INVALID_ARGUMENT;
    int n = 0;
    if (cudaGetDeviceCount(&n) != cudaSuccess) {
        *out_count = 0;
        return STARK_B200_DEVICE_FAILURE;
    }
    *out_count = n;
    return STARK_B200_OK;
}

stark_b200_status stark_b200_device_memory(uint64_t *out_free_bytes, uint64_t *out_total_bytes) {
    if (!out_free_bytes || !out_total_bytes) return STARK_B200_INVALID_ARGUMENT;
    size_t free_bytes = 0, total_bytes = 0;
    SB_CUDA(cudaMemGetInfo(&free_bytes, &total_bytes));
    *out_free_bytes = free_bytes;
    *out_total_bytes = total_bytes;
    return STARK_B200_OK;
}

stark_b200_status stark_b200_set_device(int32_t device) {
    SB_CUDA(cudaSetDevice(device));
    return STARK_B200_OK;
}

stark_b200_status stark_b200_device_malloc(void **out_ptr, size_t bytes) {
    if (!out_ptr) return STARK_B200_INVALID_ARGUMENT;
    *out_ptr = nullptr;
    SB_CUDA(cudaMalloc(out_ptr, bytes ? bytes : 1));
    return STARK_B200_OK;
}

stark_b200_status stark_b200_device_free(void *ptr) {
    SB_CUDA(cudaFree(ptr));
    return STARK_B200_OK;
}

stark_b200_status stark_b200_memcpy_h2d(void *dst, const void *src, size_t bytes, void *stream) {
    SB_CUDA(cudaMemcpyAsync(dst, src, bytes, cudaMemcpyHostToDevice, (cudaStream_t)stream));
    return STARK_B200_OK;
}

stark_b200_status stark_b200_memcpy_d2h(void *dst, const void *src, size_t bytes, void *stream) {
    SB_CUDA(cudaMemcpyAsync(dst, src, bytes, cudaMemcpyDeviceToHost, (cudaStream_t)stream));
    return STARK_B200_OK;
}

stark_b200_status stark_b200_stream_synchronize(void *stream) {
    SB_CUDA(cudaStreamSynchronize((cudaStream_t)stream));
    return STARK_B200_OK;
}

stark_b200_status stark_b200_take_device_error(uint32_t *out_word) {
    if (!out_word) return STARK_B200_INVALID_ARGUMENT;
    DeviceContext *ctx = device_context();
    if (!ctx) return STARK_B200_DEVICE_FAILURE;
    SB_CUDA(cudaMemcpy(out_word, ctx->error_word, 4, cudaMemcpyDeviceToHost));
    if (*out_word) SB_CUDA(cudaMemset(ctx->error_word, 0, 4));
    return STARK_B200_OK;
}

}  // extern "C"
