// extern "C" entry points of the session surface every model family shares: finalize, reset, prompt, step, read-outs,
// sampling, rewind, information.
#include <vector>

#include "model.cuh"
#include "tunables.cuh"

using namespace sb;

namespace {

inline Model *M(stark_b200_model *m) { return reinterpret_cast<Model *>(m); }

__global__ void bf16_to_f32_kernel(const uint16_t *in, float *out, uint32_t n) {
    for (uint32_t i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x)
        out[i] = bf16_bits_to_f32(in[i]);
}

// Temporary device mirrors of host buffers for the per-operator calls.
struct Staged {
    std::vector<void *> ptrs;
    ~Staged() {
        for (void *p : ptrs) cudaFree(p);
    }
    template <typename T>
    stark_b200_status in(const T *host, size_t count, T **dev) {
        *dev = nullptr;
        SB_CUDA(cudaMalloc(dev, count * sizeof(T) ? count * sizeof(T) : 1));
        ptrs.push_back(*dev);
        if (host) SB_CUDA(cudaMemcpy(*dev, host, count * sizeof(T), cudaMemcpyHostToDevice));
        return STARK_B200_OK;
    }
};

#define SB_TRY(expr)                                \
    do {                                            \
        stark_b200_status _s = (expr);              \
        if (_s != STARK_B200_OK) return _s;         \
    } while (0)

}  // namespace

extern "C" {

stark_b200_status stark_b200_op_sample(const void *logits, uint32_t vocab, uint32_t io_type,
                                       const stark_b200_sampling *params, uint32_t *out_token, uint32_t location,
                                       void *stream) {
    if (!logits || !params || !out_token || io_type > STARK_B200_F32) return STARK_B200_INVALID_ARGUMENT;
    if (params->struct_size != sizeof(stark_b200_sampling)) return STARK_B200_ABI_MISMATCH;
    SB_TRY(sampling_validate(*params, vocab));
    cudaStream_t s = (cudaStream_t)stream;
    Staged st;
    const uint8_t *din = static_cast<const uint8_t *>(logits);
    if (location == STARK_B200_HOST) {
        uint8_t *copy;
        SB_TRY(st.in(static_cast<const uint8_t *>(logits), (size_t)vocab * (io_type == STARK_B200_F32 ? 4u : 2u), &copy));
        din = copy;
    }
    uint8_t *scratch;
    SB_TRY(st.in((const uint8_t *)nullptr, sampling_scratch_bytes(vocab) + 16u, &scratch));
    uint32_t *out = reinterpret_cast<uint32_t *>(scratch + sampling_scratch_bytes(vocab));
    SB_TRY(sampling_launch(din, io_type, vocab, *params, scratch, out, s));
    SB_CUDA(cudaMemcpyAsync(out_token, out, 4, cudaMemcpyDeviceToHost, s));
    SB_CUDA(cudaStreamSynchronize(s));
    return STARK_B200_OK;
}

stark_b200_status stark_b200_model_finalize(stark_b200_model *model) {
    if (!model) return STARK_B200_INVALID_ARGUMENT;
    return model_finalize(M(model));
}

stark_b200_status stark_b200_destroy(stark_b200_model **model) {
    if (!model) return STARK_B200_INVALID_ARGUMENT;
    if (*model) {
        cudaStreamSynchronize(M(*model)->stream);
        delete M(*model);
        *model = nullptr;
    }
    return STARK_B200_OK;
}

stark_b200_status stark_b200_reset(stark_b200_model *model) {
    if (!model) return STARK_B200_INVALID_ARGUMENT;
    if (M(model)->fenced) return STARK_B200_RELOAD_REQUIRED;
    return model_reset(M(model));
}

stark_b200_status stark_b200_drain(stark_b200_model *model) {
    if (!model) return STARK_B200_INVALID_ARGUMENT;
    return model_drain(M(model));
}

stark_b200_status stark_b200_cancel(stark_b200_model *model) {
    if (!model) return STARK_B200_INVALID_ARGUMENT;
    M(model)->cancel_requested = true;
    return STARK_B200_OK;
}

stark_b200_status stark_b200_prefill(stark_b200_model *model, const uint32_t *token_ids, size_t count) {
    if (!model || !token_ids) return STARK_B200_INVALID_ARGUMENT;
    return model_prefill(M(model), token_ids, count);
}

stark_b200_status stark_b200_prefill_rows(stark_b200_model *model, const uint32_t *token_ids, size_t count,
                                          const uint32_t *wanted, size_t wanted_count, float *dst) {
    if (!model || !token_ids || (wanted_count && (!wanted || !dst))) return STARK_B200_INVALID_ARGUMENT;
    return model_prefill_rows(M(model), token_ids, count, wanted, wanted_count, dst);
}

stark_b200_status stark_b200_step(stark_b200_model *model, uint32_t token_id) {
    if (!model) return STARK_B200_INVALID_ARGUMENT;
    return model_step(M(model), token_id, false);
}

stark_b200_status stark_b200_readout_f32(stark_b200_model *model, float *dst, size_t count) {
    if (!model || !dst) return STARK_B200_INVALID_ARGUMENT;
    return model_readout_f32(M(model), dst, count);
}

stark_b200_status stark_b200_readout_bf16(stark_b200_model *model, uint16_t *dst, size_t count) {
    if (!model || !dst) return STARK_B200_INVALID_ARGUMENT;
    return model_readout_bf16(M(model), dst, count);
}

stark_b200_status stark_b200_readout_logprobs_f32(stark_b200_model *model, float *dst, size_t count) {
    if (!model || !dst) return STARK_B200_INVALID_ARGUMENT;
    Model *m = M(model);
    if (!m->has_logits) return STARK_B200_INVALID_STATE;
    if (m->tp.size > 1u) return STARK_B200_UNSUPPORTED;  // a shard's logits do not normalise alone
    if (count != m->cfg.vocab) return STARK_B200_INVALID_ARGUMENT;
    Staged st;
    float *df;
    double *dd;
    SB_TRY(st.in((const double *)nullptr, count, &dd));
    if (m->logits_f32) {
        df = m->logits_f32;
    } else {
        SB_TRY(st.in((const float *)nullptr, count, &df));
        bf16_to_f32_kernel<<<148, 256, 0, m->stream>>>(m->logits, df, (uint32_t)count);
    }
    SB_TRY(log_softmax_launch(df, dd, (uint32_t)count, nullptr, m->stream));
    std::vector<double> host(count);
    SB_CUDA(cudaMemcpyAsync(host.data(), dd, count * 8, cudaMemcpyDeviceToHost, m->stream));
    SB_CUDA(cudaStreamSynchronize(m->stream));
    for (size_t i = 0; i < count; ++i) dst[i] = (float)host[i];
    return STARK_B200_OK;
}

stark_b200_status stark_b200_sample(stark_b200_model *model, const stark_b200_sampling *params, uint32_t *out_token) {
    if (!model || !params || !out_token) return STARK_B200_INVALID_ARGUMENT;
    if (params->struct_size != sizeof(stark_b200_sampling)) return STARK_B200_ABI_MISMATCH;
    Model *m = M(model);
    if (!m->has_logits) return STARK_B200_INVALID_STATE;
    if (m->tp.size > 1u) return STARK_B200_UNSUPPORTED;
    SB_TRY(sampling_validate(*params, m->cfg.vocab));
    if (!m->sample_scratch) SB_CUDA(cudaMalloc(&m->sample_scratch, sampling_scratch_bytes(m->cfg.vocab) + 16u));
    // the token lands behind the working arrays
    uint32_t *out = reinterpret_cast<uint32_t *>(static_cast<uint8_t *>(m->sample_scratch) +
                                                 sampling_scratch_bytes(m->cfg.vocab));
    SB_TRY(m->logits_f32 ? sampling_launch(m->logits_f32, STARK_B200_F32, m->cfg.vocab, *params, m->sample_scratch, out, m->stream)
                         : sampling_launch(m->logits, STARK_B200_BF16, m->cfg.vocab, *params, m->sample_scratch, out, m->stream));
    SB_CUDA(cudaMemcpyAsync(out_token, out, 4, cudaMemcpyDeviceToHost, m->stream));
    SB_CUDA(cudaStreamSynchronize(m->stream));
    return STARK_B200_OK;
}

stark_b200_status stark_b200_argmax(stark_b200_model *model, uint32_t *out_token) {
    if (!model || !out_token) return STARK_B200_INVALID_ARGUMENT;
    return model_next_token(M(model), out_token);
}

stark_b200_status stark_b200_generate_greedy(stark_b200_model *model, uint32_t steps, uint32_t *out_tokens) {
    if (!model || !out_tokens) return STARK_B200_INVALID_ARGUMENT;
    return model_generate_greedy(M(model), steps, out_tokens);
}

stark_b200_status stark_b200_rewind(stark_b200_model *model, uint64_t position) {
    if (!model) return STARK_B200_INVALID_ARGUMENT;
    return model_rewind(M(model), position);
}

stark_b200_status stark_b200_set_tunable(const char *name, uint32_t value) {
    return set_tunable(name, value) ? STARK_B200_OK : STARK_B200_INVALID_ARGUMENT;
}

stark_b200_status stark_b200_model_recapture(stark_b200_model *model) {
    if (!model) return STARK_B200_INVALID_ARGUMENT;
    if (M(model)->tp.size > 1u) return STARK_B200_UNSUPPORTED;
    return model_recapture(M(model));
}

stark_b200_status stark_b200_model_stream(stark_b200_model *model, void **out_stream) {
    if (!model || !out_stream) return STARK_B200_INVALID_ARGUMENT;
    *out_stream = (void *)M(model)->stream;
    return STARK_B200_OK;
}

stark_b200_status stark_b200_read_trace(stark_b200_model *model, uint64_t *dst, size_t count) {
    if (!model || !dst) return STARK_B200_INVALID_ARGUMENT;
    return model_read_trace(M(model), reinterpret_cast<unsigned long long *>(dst), count);
}

stark_b200_status stark_b200_get_info(stark_b200_model *model, stark_b200_info *info) {
    if (!model || !info) return STARK_B200_INVALID_ARGUMENT;
    if (info->struct_size != sizeof(stark_b200_info) || info->abi_version != STARK_B200_ABI_VERSION)
        return STARK_B200_ABI_MISMATCH;
    Model *m = M(model);
    info->vocab_size = m->cfg.vocab;
    info->prefill_chunk_tokens = 1024;
    info->context_tokens = m->cfg.context_tokens;
    info->position = m->position;
    info->capabilities = STARK_B200_CAP_FULL_F32_READOUT | STARK_B200_CAP_SERIAL_DECODE |
                         STARK_B200_CAP_PREFIX_REWIND | STARK_B200_CAP_DEVICE_GREEDY;
    info->fenced = m->fenced ? 1u : 0u;
    info->launches_per_step = m->step_launches;
    m->family->sizes(m, &info->weight_bytes, &info->kv_bytes_per_token);
    info->launches_issued = m->launches_issued;
    info->trace_slots = m->trace ? m->trace_slots : 0u;
    info->persistent = m->use_mega ? 1u : 0u;
    return STARK_B200_OK;
}

}  // extern "C"
